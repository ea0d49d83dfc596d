// Recurrences whose state is a sum of outer products k v^T per head, walked token by token in
// float32 from the state the row's slot holds:
//
//   wkv_scan      a decay per key channel and a bonus for the current token:
//                 o_t = S_(t-1)^T r_t + (sum_d r_t[d] u[d] k_t[d]) v_t;  S_t = diag(w_t) S_(t-1) + k_t v_t^T
//   mlstm_scan    exponential gates with a running maximum m (from 0) and a normalizer n:
//                 i = c tanh((i~ + bi) / c),  f = log sigmoid(c tanh((f~ + bf) / c));
//                 m_t = max(f + m_(t-1), i);  S_t = e^(f + m_(t-1) - m_t) S_(t-1) + e^(i - m_t) k_t v_t^T,
//                 n_t likewise with k_t alone;  out = S_t^T q_t,  den = max(|n_t . q_t|, e^(-m_t)) + 1e-6
//                 (the division is the next kernel's, which norms each head anyway).  n is kept as
//                 one more column of S, whose value is always 1.
//   wkv_decay     w = exp(-exp(w0 + W2 tanh(t1))) per token and channel, W2 through a small rank
//
// The scan: a block owns (row, head, a tile of columns); LD neighbouring lanes share a pair of
// columns and hold its state elements d = 4 (l + LD i) .. + 3 in registers, so that what a lane
// reads of q, k and the decays from shared memory (16 bytes at a time) serves two columns.  Tokens
// come in chunks through two cp.async buffers, four tokens' sums side by side: their eight numbers
// are summed over the lanes by halving (each step sends what the partner keeps), 4 + 2 + 1
// shuffles and one more for every doubling of LD beyond 8.  A sum's tree does not depend on the
// chunk, so the cut of a sequence changes nothing but the order of nothing.
// State [slots][heads][columns][D]: a column's elements are contiguous.  Every column keeps its own
// copy of the running maximum ([slots][heads][columns]), so no block reads what another writes.
// Tokens are packed row after row (row b: tokens cu_seqlens[b] .. cu_seqlens[b + 1]).
#include "common.cuh"

#define OS_THREADS 128
#define OS_TU 4              // tokens whose sums are formed side by side
#define OS_MAX_D 256

struct OuterScanArgs {
    const float* r;          // read vectors (r or q): r[t * r_width + r_off + head * D + d]
    const float* k;
    const float* v;          // v[t * v_width + v_off + head * Dv + j]
    const float* w;          // wkv: decays w[t * w_width + w_off + head * D + d]
    const float* u;          // wkv: bonus [heads][D]
    const float* gates;      // mlstm: raw gates, gates[t * gate_width + i_off + head], .. f_off ..
    const float* i_bias;     // [heads]
    const float* f_bias;     // [heads]
    float* state;            // [slots][heads][columns][D], columns Dv (wkv) or Dv + 1 (mlstm)
    float* maxima;           // mlstm: [slots][heads][Dv + 1]
    const int* cu_seqlens;
    const int* slots;
    float* out;              // [tokens][heads * Dv]
    float* den;              // mlstm: [tokens][heads]
    long long r_width, k_width, v_width, w_width, gate_width;
    int r_off, k_off, v_off, w_off, i_off, f_off;
    int n_rows, heads, D, Dv;
    float cap, r_scale;      // mlstm: cap of the gates; factor on q
};

__device__ __forceinline__ void os_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;"
                 ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void os_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;"
                 ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Sums the 8 numbers of every lane over groups of LD lanes.  The lane with index l of its group gets
// number l / (LD / 8), complete.
template <int LD>
__device__ __forceinline__ float os_reduce8(float (&a)[8], int l) {
    int o = LD / 2;
#pragma unroll
    for (int half = 4; half >= 1; half >>= 1, o >>= 1) {
        const bool up = (l & o) != 0;
#pragma unroll
        for (int j = 0; j < half; ++j) {
            const float send = up ? a[j] : a[j + half];
            const float keep = up ? a[j + half] : a[j];
            a[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
    float s = a[0];
#pragma unroll
    for (; o >= 1; o >>= 1) s += __shfl_xor_sync(0xffffffffu, s, o);
    return s;
}

// One token on this thread's two columns: acc += (state read with r), state updated.
template <int ND4, bool WKV>
__device__ __forceinline__ void os_token(float4 (&S0)[ND4], float4 (&S1)[ND4], const float4* r4,
                                         const float4* k4, const float4* w4, float keep, float v0,
                                         float v1, int step, float& acc0, float& acc1) {
    float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
#pragma unroll
    for (int i = 0; i < ND4; ++i) {
        const float4 rr = r4[i * step], kk = k4[i * step];
        if (WKV) {
            const float4 ww = w4[i * step];
            a0 = fmaf(rr.x, S0[i].x, a0); b0 = fmaf(rr.y, S0[i].y, b0);
            a0 = fmaf(rr.z, S0[i].z, a0); b0 = fmaf(rr.w, S0[i].w, b0);
            a1 = fmaf(rr.x, S1[i].x, a1); b1 = fmaf(rr.y, S1[i].y, b1);
            a1 = fmaf(rr.z, S1[i].z, a1); b1 = fmaf(rr.w, S1[i].w, b1);
            S0[i].x = fmaf(ww.x, S0[i].x, kk.x * v0); S1[i].x = fmaf(ww.x, S1[i].x, kk.x * v1);
            S0[i].y = fmaf(ww.y, S0[i].y, kk.y * v0); S1[i].y = fmaf(ww.y, S1[i].y, kk.y * v1);
            S0[i].z = fmaf(ww.z, S0[i].z, kk.z * v0); S1[i].z = fmaf(ww.z, S1[i].z, kk.z * v1);
            S0[i].w = fmaf(ww.w, S0[i].w, kk.w * v0); S1[i].w = fmaf(ww.w, S1[i].w, kk.w * v1);
        } else {
            S0[i].x = fmaf(keep, S0[i].x, kk.x * v0); S1[i].x = fmaf(keep, S1[i].x, kk.x * v1);
            S0[i].y = fmaf(keep, S0[i].y, kk.y * v0); S1[i].y = fmaf(keep, S1[i].y, kk.y * v1);
            S0[i].z = fmaf(keep, S0[i].z, kk.z * v0); S1[i].z = fmaf(keep, S1[i].z, kk.z * v1);
            S0[i].w = fmaf(keep, S0[i].w, kk.w * v0); S1[i].w = fmaf(keep, S1[i].w, kk.w * v1);
            a0 = fmaf(rr.x, S0[i].x, a0); b0 = fmaf(rr.y, S0[i].y, b0);
            a0 = fmaf(rr.z, S0[i].z, a0); b0 = fmaf(rr.w, S0[i].w, b0);
            a1 = fmaf(rr.x, S1[i].x, a1); b1 = fmaf(rr.y, S1[i].y, b1);
            a1 = fmaf(rr.z, S1[i].z, a1); b1 = fmaf(rr.w, S1[i].w, b1);
        }
    }
    acc0 = a0 + b0;
    acc1 = a1 + b1;
}

__device__ __forceinline__ float os_soft_cap(float z, float cap) { return cap * tanhf(z / cap); }

// LD: lanes that share a pair of columns; ND4: float4 groups of a column a lane holds (D <= 4 LD ND4);
// tc: tokens of a chunk (mlstm: at most 32)
template <int LD, int ND4, bool WKV>
__global__ void __launch_bounds__(OS_THREADS) outer_scan_kernel(OuterScanArgs a, int tc) {
    pdl_launch_dependents();
    constexpr int DP = 4 * LD * ND4;                   // padded key size
    constexpr int TV = 2 * (OS_THREADS / LD);          // columns of a block
    constexpr int NVEC = WKV ? 3 : 2;                  // vectors staged per token: r, k (and decays)
    extern __shared__ __align__(16) float os_smem[];
    const int buf_floats = tc * (NVEC * DP + TV) + (WKV ? 0 : 2 * tc);   // r k (w) | v | raw i, f
    float* o_s = os_smem + 2 * buf_floats;             // [tc][TV]
    float* keep_s = o_s + tc * TV;                     // [tc] mlstm: decay of the state; wkv: r . (u k)
    float* add_s = keep_s + tc;                        // [tc] mlstm: factor on the new term
    float* floor_s = add_s + tc;                       // [tc] mlstm: e^(-m)
    const int D = a.D, Dv = a.Dv;
    const int cols = WKV ? Dv : Dv + 1;
    const int tiles = (cols + TV - 1) / TV;
    const int h = blockIdx.x / tiles, tile = blockIdx.x - h * tiles;
    const int b = blockIdx.y;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int l = tid % LD, c = tid / LD;              // lane of the pair's group; pair of columns
    const int j0 = tile * TV, n_cols = min(TV, cols - j0);
    const bool live0 = 2 * c < n_cols, live1 = 2 * c + 1 < n_cols;
    const int t0 = a.cu_seqlens[b], n_b = a.cu_seqlens[b + 1] - t0;
    const int slot = a.slots[b];
    // (a row of a tensor may start anywhere: 16-byte copies only where all of them start on 16 bytes)
    const bool vec = (D & 3) == 0 &&
                     ((a.r_width | a.k_width | a.w_width | (long long)(a.r_off | a.k_off | a.w_off)) & 3) == 0 &&
                     (((uintptr_t)a.r | (uintptr_t)a.k | (uintptr_t)a.w) & 15) == 0;
    if (DP > D) {                                      // the copies never touch the padding
        const int pad = DP - D;
        for (int i = tid; i < 2 * tc * NVEC * pad; i += OS_THREADS) {
            const int row = i / pad, d = D + i - row * pad;
            const int buf = row / (tc * NVEC), rr = row - buf * tc * NVEC;
            os_smem[buf * buf_floats + rr * DP + d] = 0.0f;
        }
    }
    float ib = 0.f, fb = 0.f;
    if (!WKV) { ib = a.i_bias[h]; fb = a.f_bias[h]; }
    pdl_wait();
    if (n_b <= 0) return;

    auto fetch = [&](int c0, int buf) {
        const int nc = min(tc, n_b - c0);
        float* r_s = os_smem + buf * buf_floats;
        float* k_s = r_s + tc * DP;
        float* w_s = k_s + tc * DP;                    // (wkv)
        float* v_s = r_s + tc * NVEC * DP;
        if (vec) {
            const int qn = D >> 2;
            for (int i = tid; i < nc * qn; i += OS_THREADS) {
                const int tt = i / qn, d = (i - tt * qn) << 2;
                const size_t t = (size_t)(t0 + c0 + tt);
                os_cp16(r_s + tt * DP + d, a.r + t * a.r_width + a.r_off + h * D + d);
                os_cp16(k_s + tt * DP + d, a.k + t * a.k_width + a.k_off + h * D + d);
                if (WKV) os_cp16(w_s + tt * DP + d, a.w + t * a.w_width + a.w_off + h * D + d);
            }
        } else {
            for (int i = tid; i < nc * D; i += OS_THREADS) {
                const int tt = i / D, d = i - tt * D;
                const size_t t = (size_t)(t0 + c0 + tt);
                os_cp4(r_s + tt * DP + d, a.r + t * a.r_width + a.r_off + h * D + d);
                os_cp4(k_s + tt * DP + d, a.k + t * a.k_width + a.k_off + h * D + d);
                if (WKV) os_cp4(w_s + tt * DP + d, a.w + t * a.w_width + a.w_off + h * D + d);
            }
        }
        for (int i = tid; i < nc * n_cols; i += OS_THREADS) {
            const int tt = i / n_cols, cc = i - tt * n_cols;
            if (WKV || j0 + cc < Dv)
                os_cp4(v_s + tt * TV + cc, a.v + (size_t)(t0 + c0 + tt) * a.v_width + a.v_off + (size_t)h * Dv + j0 + cc);
            else
                v_s[tt * TV + cc] = 1.0f;              // the normalizer's column
        }
        if (!WKV) {
            float* g_s = v_s + tc * TV;
            for (int i = tid; i < 2 * nc; i += OS_THREADS) {
                const int tt = i >> 1;
                os_cp4(g_s + (i & 1) * tc + tt,
                       a.gates + (size_t)(t0 + c0 + tt) * a.gate_width + ((i & 1) ? a.f_off : a.i_off) + h);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    fetch(0, 0);

    float* st0 = a.state + (((size_t)slot * a.heads + h) * cols + j0 + (live0 ? 2 * c : 0)) * D;
    float* st1 = live1 ? st0 + D : st0;
    float4 S0[ND4], S1[ND4];
    const bool vec_state = (D & 3) == 0;
    auto get = [&](const float* p, int d, bool ok) {
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (ok) {
            if (vec_state) {
                if (d < D) x = *reinterpret_cast<const float4*>(p + d);
            } else {
                if (d < D) x.x = p[d];
                if (d + 1 < D) x.y = p[d + 1];
                if (d + 2 < D) x.z = p[d + 2];
                if (d + 3 < D) x.w = p[d + 3];
            }
        }
        return x;
    };
#pragma unroll
    for (int i = 0; i < ND4; ++i) {
        S0[i] = get(st0, 4 * (l + LD * i), live0);
        S1[i] = get(st1, 4 * (l + LD * i), live1);
    }
    float m_run = 0.f;                                 // (warp 0) the running maximum
    if (!WKV) m_run = a.maxima[((size_t)slot * a.heads + h) * cols + j0];

    for (int c0 = 0, buf = 0; c0 < n_b; c0 += tc, buf ^= 1) {
        const int nc = min(tc, n_b - c0);
        if (c0 + tc < n_b) {
            fetch(c0 + tc, buf ^ 1);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();                 // the chunk has arrived; the last chunk's outputs are written
        const float* r_s = os_smem + buf * buf_floats;
        const float* k_s = r_s + tc * DP;
        const float* w_s = k_s + tc * DP;
        const float* v_s = r_s + tc * NVEC * DP;
        if (WKV) {
            // r . (u k): what the current token's own value is multiplied by
            for (int tt = warp; tt < nc; tt += OS_THREADS / 32) {
                float s = 0.f;
                for (int d = lane; d < D; d += 32)
                    s = fmaf(r_s[tt * DP + d] * a.u[h * D + d], k_s[tt * DP + d], s);
                s = warp_sum(s);
                if (lane == 0) keep_s[tt] = s;
            }
        } else if (warp == 0) {
            // the gates of the chunk's tokens, a lane each; the maxima by a scan in which a stretch
            // of tokens is the pair (sum of f, largest i + the f's after it)
            const float* g_s = v_s + tc * TV;
            const bool mine = lane < nc;
            const float li = mine ? os_soft_cap(g_s[lane] + ib, a.cap) : -INFINITY;
            const float zf = mine ? os_soft_cap(g_s[tc + lane] + fb, a.cap) : 0.f;
            const float lf = mine ? fminf(zf, 0.f) - log1pf(expf(-fabsf(zf))) : 0.f;
            float F = lf, M = li;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float pF = __shfl_up_sync(0xffffffffu, F, o), pM = __shfl_up_sync(0xffffffffu, M, o);
                if (lane >= o) { M = fmaxf(pM + F, M); F = pF + F; }
            }
            const float m_t = fmaxf(F + m_run, M);
            float before = __shfl_up_sync(0xffffffffu, m_t, 1);
            if (lane == 0) before = m_run;
            if (mine) {
                // (m_t is often lf + before, rounded: in this order the difference is exact, so what m_t lost
                // in rounding stays in the state's factor instead of adding up token by token)
                keep_s[lane] = expf((before - m_t) + lf);
                add_s[lane] = expf(li - m_t);
                floor_s[lane] = expf(-m_t);
            }
            m_run = __shfl_sync(0xffffffffu, m_t, nc - 1);
        }
        if (!WKV) __syncthreads();       // (wkv reads its factors after the tokens, behind a barrier)
        int tt = 0;
        for (; tt + OS_TU <= nc; tt += OS_TU) {
            float acc[2 * OS_TU];
#pragma unroll
            for (int u = 0; u < OS_TU; ++u) {
                const int t = tt + u;
                const float2 vv = *reinterpret_cast<const float2*>(v_s + t * TV + 2 * c);
                float v0 = live0 ? vv.x : 0.f, v1 = live1 ? vv.y : 0.f, keep = 0.f;
                if (!WKV) { keep = keep_s[t]; v0 *= add_s[t]; v1 *= add_s[t]; }
                os_token<ND4, WKV>(S0, S1, reinterpret_cast<const float4*>(r_s + t * DP) + l,
                                   reinterpret_cast<const float4*>(k_s + t * DP) + l,
                                   reinterpret_cast<const float4*>(w_s + t * DP) + l, keep, v0, v1, LD,
                                   acc[2 * u], acc[2 * u + 1]);
            }
            const float sum = os_reduce8<LD>(acc, l);
            constexpr int PER = LD / 8;                // lanes that hold the same sum
            if (l % PER == 0) {
                const int i = l / PER;
                o_s[(tt + (i >> 1)) * TV + 2 * c + (i & 1)] = sum;
            }
        }
        for (; tt < nc; ++tt) {
            const float2 vv = *reinterpret_cast<const float2*>(v_s + tt * TV + 2 * c);
            float v0 = live0 ? vv.x : 0.f, v1 = live1 ? vv.y : 0.f, keep = 0.f, a0, a1;
            if (!WKV) { keep = keep_s[tt]; v0 *= add_s[tt]; v1 *= add_s[tt]; }
            os_token<ND4, WKV>(S0, S1, reinterpret_cast<const float4*>(r_s + tt * DP) + l,
                               reinterpret_cast<const float4*>(k_s + tt * DP) + l,
                               reinterpret_cast<const float4*>(w_s + tt * DP) + l, keep, v0, v1, LD, a0, a1);
#pragma unroll
            for (int o = LD / 2; o > 0; o >>= 1) {
                a0 += __shfl_xor_sync(0xffffffffu, a0, o);
                a1 += __shfl_xor_sync(0xffffffffu, a1, o);
            }
            if (l == 0) { o_s[tt * TV + 2 * c] = a0; o_s[tt * TV + 2 * c + 1] = a1; }
        }
        __syncthreads();                 // the chunk's outputs are complete; its buffer may be refilled
        for (int i = tid; i < nc * n_cols; i += OS_THREADS) {
            const int t2 = i / n_cols, cc = i - t2 * n_cols;
            const size_t t = (size_t)(t0 + c0 + t2);
            const float x = o_s[t2 * TV + cc];
            if (WKV)
                a.out[t * a.heads * Dv + (size_t)h * Dv + j0 + cc] = fmaf(keep_s[t2], v_s[t2 * TV + cc], x);
            else if (j0 + cc < Dv)
                a.out[t * a.heads * Dv + (size_t)h * Dv + j0 + cc] = x * a.r_scale;
            else
                a.den[t * a.heads + h] = fmaxf(fabsf(x * a.r_scale), floor_s[t2]) + 1e-6f;
        }
        // (the next chunk's copies go to the other buffer, and its factors are formed behind the
        // barrier at the head of the loop)
        if (WKV && c0 + tc < n_b) __syncthreads();     // its v is about to be the target of the copy after next
    }
    auto put = [&](float* p, int d, const float4& x) {
        if (vec_state) {
            if (d < D) *reinterpret_cast<float4*>(p + d) = x;
        } else {
            if (d < D) p[d] = x.x;
            if (d + 1 < D) p[d + 1] = x.y;
            if (d + 2 < D) p[d + 2] = x.z;
            if (d + 3 < D) p[d + 3] = x.w;
        }
    };
#pragma unroll
    for (int i = 0; i < ND4; ++i) {
        if (live0) put(st0, 4 * (l + LD * i), S0[i]);
        if (live1) put(st1, 4 * (l + LD * i), S1[i]);
    }
    if (!WKV && warp == 0)
        for (int i = lane; i < n_cols; i += 32) a.maxima[((size_t)slot * a.heads + h) * cols + j0 + i] = m_run;
}

template <int LD, int ND4, bool WKV>
static int os_launch(const OuterScanArgs& a, cudaStream_t stream) {
    constexpr int DP = 4 * LD * ND4, TV = 2 * (OS_THREADS / LD), NVEC = WKV ? 3 : 2;
    const int tc = DP > 128 ? 16 : 32;
    const size_t smem = (size_t)(2 * (tc * (NVEC * DP + TV) + (WKV ? 0 : 2 * tc)) + tc * TV + 3 * tc) * sizeof(float);
    static bool configured[64] = {false};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return MF_ERR_UNSUPPORTED;
    if (!configured[dev]) {
        cudaError_t e = cudaFuncSetAttribute(outer_scan_kernel<LD, ND4, WKV>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured[dev] = true;
    }
    const int cols = WKV ? a.Dv : a.Dv + 1;
    const int tiles = (cols + TV - 1) / TV;
    mf_launch(outer_scan_kernel<LD, ND4, WKV>, dim3(a.heads * tiles, a.n_rows), dim3(OS_THREADS), smem,
              stream, a, tc);
    return MF_LAUNCH_CHECK();
}

template <bool WKV>
static int os_choose(const OuterScanArgs& a, cudaStream_t stream) {
    if (a.n_rows <= 0) return 0;
    if (a.D < 1 || a.D > OS_MAX_D || a.Dv < 1 || a.heads < 1 || a.n_rows > 65535) return MF_ERR_UNSUPPORTED;
    if (((uintptr_t)a.state & 15) != 0) return MF_ERR_UNSUPPORTED;
    if (a.D <= 32) return os_launch<8, 1, WKV>(a, stream);
    if (a.D <= 64) return os_launch<16, 1, WKV>(a, stream);
    if (a.D <= 128) return os_launch<16, 2, WKV>(a, stream);
    return os_launch<32, 2, WKV>(a, stream);
}

extern "C" int mf_wkv_scan(const OuterScanArgs* args, cudaStream_t stream) {
    return os_choose<true>(*args, stream);
}
extern "C" int mf_mlstm_scan(const OuterScanArgs* args, cudaStream_t stream) {
    if (!(args->cap > 0.0f)) return MF_ERR_ARGUMENT;
    return os_choose<false>(*args, stream);
}

// ------------------------------------------------------------------------------------------
// out[t][c] = exp(-exp(w0[c] + sum_r w2t[r][c] tanh(t1[t][r]))): a thread per channel, WD_T tokens a
// block, whose tanh(t1) lie in shared memory.
// ------------------------------------------------------------------------------------------
#define WD_T 16

template <int NT>
__global__ void __launch_bounds__(128)
wkv_decay_kernel(const float* __restrict__ t1, long long t1_width, const float* __restrict__ w2t,
                 const float* __restrict__ w0, float* __restrict__ out, int n_tokens, int rank, int channels) {
    pdl_prologue();
    extern __shared__ float wd_s[];                    // [NT][rank]
    const int first = blockIdx.y * NT, nt = min(NT, n_tokens - first);
    for (int i = threadIdx.x; i < NT * rank; i += blockDim.x) {
        const int t = i / rank, r = i - t * rank;
        wd_s[i] = t < nt ? tanhf(t1[(size_t)(first + t) * t1_width + r]) : 0.f;
    }
    __syncthreads();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    float acc[NT];
    const float base = w0[c];
#pragma unroll
    for (int t = 0; t < NT; ++t) acc[t] = base;
#pragma unroll 4
    for (int r = 0; r < rank; ++r) {
        const float w = w2t[(size_t)r * channels + c];
#pragma unroll
        for (int t = 0; t < NT; ++t) acc[t] = fmaf(w, wd_s[t * rank + r], acc[t]);
    }
#pragma unroll
    for (int t = 0; t < NT; ++t)
        if (t < nt) out[(size_t)(first + t) * channels + c] = expf(-expf(acc[t]));
}

extern "C" int mf_wkv_decay(const float* t1, long long t1_width, const float* w2t, const float* w0,
                            float* out, int n_tokens, int rank, int channels, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rank < 1 || channels < 1 || (size_t)rank * WD_T * sizeof(float) > 48 * 1024) return MF_ERR_UNSUPPORTED;
    const int cb = (channels + 127) / 128;
    if (n_tokens <= 64) {
        if ((n_tokens + 1) / 2 > 65535) return MF_ERR_UNSUPPORTED;
        mf_launch(wkv_decay_kernel<2>, dim3(cb, (n_tokens + 1) / 2), dim3(128), (size_t)rank * 2 * sizeof(float),
                  stream, t1, t1_width, w2t, w0, out, n_tokens, rank, channels);
    } else {
        if ((n_tokens + WD_T - 1) / WD_T > 65535) return MF_ERR_UNSUPPORTED;
        mf_launch(wkv_decay_kernel<WD_T>, dim3(cb, (n_tokens + WD_T - 1) / WD_T), dim3(128),
                  (size_t)rank * WD_T * sizeof(float), stream, t1, t1_width, w2t, w0, out, n_tokens, rank, channels);
    }
    return MF_LAUNCH_CHECK();
}
