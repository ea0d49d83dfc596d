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
//   gla_scan      a decay per key channel, the current token's own pair included in what it reads:
//                 S_t = diag(w_t) S_(t-1) + k_t v_t^T;  o_t = S_t^T q_t
//   wkv_decay     w = exp(-exp(w0 + W2 tanh(t1))) per token and channel, W2 through a small rank
//   sigmoid_decay w = sigmoid(w0 + W2 t1)^(1 / tau), likewise
//
// The scan: a block owns (row, head, a tile of columns).  Four warps walk the tokens: LD neighbouring
// lanes share a pair of columns and hold its state elements d = 4 (l + LD i) .. + 3 in registers, so
// that what a lane reads of q, k and the decays from shared memory (16 bytes at a time) serves two
// columns.  The sums of eight tokens (16 numbers a lane) are formed side by side and added over the
// lanes by halving: each step sends what the partner keeps, 8 + 4 + 2 + 1 shuffles for all of them.  A
// sum's tree does not depend on how the tokens are grouped.  Four more warps do what is not the
// chain: they keep a ring of four chunks of tokens filled by cp.async, two chunks ahead, and prepare
// each (wkv: r . (u k); mlstm: gates and maxima), handing chunks over and taking them back through
// named barriers.
// State [slots][heads][columns][D]: a column's elements are contiguous.  Every column keeps its own
// copy of the running maximum ([slots][heads][columns]), so no block reads what another writes.
// Tokens are packed row after row (row b: tokens cu_seqlens[b] .. cu_seqlens[b + 1]).
#include "common.cuh"

#define OS_THREADS 128       // the threads that walk the tokens
#define OS_FEED 4            // warps that feed them
#define OS_TU 8              // tokens whose sums are formed side by side
#define OS_TC 16             // tokens of a chunk
#define OS_STAGES 4
#define OS_MAX_D 256

// the recurrences; which of them have a decay per key channel, a bonus, gates with a running maximum
enum OuterMode { OS_WKV = 0, OS_MLSTM = 1, OS_GLA = 2 };
template <int MODE> struct OuterTraits {
    static constexpr bool DECAYS = MODE != OS_MLSTM, BONUS = MODE == OS_WKV, GATES = MODE == OS_MLSTM;
};

struct OuterScanArgs {
    const float* r;          // read vectors (r or q): r[t * r_width + r_off + head * D + d]
    const float* k;
    const float* v;          // v[t * v_width + v_off + head * Dv + j]
    const float* w;          // wkv, gla: decays w[t * w_width + w_off + head * D + d]
    const float* u;          // wkv: bonus [heads][D]
    const float* gates;      // mlstm: raw gates, gates[t * gate_width + i_off + head], .. f_off ..
    const float* i_bias;     // [heads]
    const float* f_bias;     // [heads]
    float* state;            // [slots][heads][columns][D], columns Dv or Dv + 1 (mlstm)
    float* maxima;           // mlstm: [slots][heads][Dv + 1]
    const int* cu_seqlens;
    const int* slots;
    float* out;              // [tokens][heads * Dv]
    float* den;              // mlstm: [tokens][heads]
    long long r_width, k_width, v_width, w_width, gate_width;
    int r_off, k_off, v_off, w_off, i_off, f_off;
    int n_rows, heads, D, Dv;
    float cap, r_scale;      // mlstm: cap of the gates; mlstm, gla: factor on q
};

__device__ __forceinline__ void os_cp4(float* dst, const float* src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;"
                 ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void os_cp16(float* dst, const float* src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;"
                 ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// Sums the 16 numbers of every lane over groups of LD lanes.  The lane with index l of its group gets
// LD 8: numbers 2 l and 2 l + 1 (in a[0], a[1]); LD 16: number l; LD 32: number l / 2.
template <int LD>
__device__ __forceinline__ void os_reduce16(float (&a)[16], int l) {
    int o = LD / 2;
#pragma unroll
    for (int half = 8; half >= 1; half >>= 1, o >>= 1) {
        if (o == 0) break;
        const bool up = (l & o) != 0;
#pragma unroll
        for (int j = 0; j < half; ++j) {
            const float send = up ? a[j] : a[j + half];
            const float keep = up ? a[j + half] : a[j];
            a[j] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
    if (LD == 32) a[0] += __shfl_xor_sync(0xffffffffu, a[0], 1);
}

// named barriers of the hand-over (0 is __syncthreads): all eight warps take part
__device__ __forceinline__ void os_bar_sync(int id) {
    asm volatile("bar.sync %0, %1;" ::"r"(id), "n"(OS_THREADS + 32 * OS_FEED) : "memory");
}
__device__ __forceinline__ void os_bar_arrive(int id) {
    asm volatile("bar.arrive %0, %1;" ::"r"(id), "n"(OS_THREADS + 32 * OS_FEED) : "memory");
}
#define OS_FULL(stage) (1 + (stage))
#define OS_EMPTY(stage) (1 + OS_STAGES + (stage))

// One token on this thread's two columns: acc += (state read with r), state updated.
template <int ND4, int MODE>
__device__ __forceinline__ void os_token(float4 (&S0)[ND4], float4 (&S1)[ND4], const float4* r4,
                                         const float4* k4, const float4* w4, float keep, float v0,
                                         float v1, int step, float& acc0, float& acc1) {
    float a0 = 0.f, a1 = 0.f, b0 = 0.f, b1 = 0.f;
#pragma unroll
    for (int i = 0; i < ND4; ++i) {
        const float4 rr = r4[i * step], kk = k4[i * step];
        if (MODE == OS_GLA) {
            const float4 ww = w4[i * step];
            S0[i].x = fmaf(ww.x, S0[i].x, kk.x * v0); S1[i].x = fmaf(ww.x, S1[i].x, kk.x * v1);
            S0[i].y = fmaf(ww.y, S0[i].y, kk.y * v0); S1[i].y = fmaf(ww.y, S1[i].y, kk.y * v1);
            S0[i].z = fmaf(ww.z, S0[i].z, kk.z * v0); S1[i].z = fmaf(ww.z, S1[i].z, kk.z * v1);
            S0[i].w = fmaf(ww.w, S0[i].w, kk.w * v0); S1[i].w = fmaf(ww.w, S1[i].w, kk.w * v1);
            a0 = fmaf(rr.x, S0[i].x, a0); b0 = fmaf(rr.y, S0[i].y, b0);
            a0 = fmaf(rr.z, S0[i].z, a0); b0 = fmaf(rr.w, S0[i].w, b0);
            a1 = fmaf(rr.x, S1[i].x, a1); b1 = fmaf(rr.y, S1[i].y, b1);
            a1 = fmaf(rr.z, S1[i].z, a1); b1 = fmaf(rr.w, S1[i].w, b1);
        } else if (MODE == OS_WKV) {
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
// tc: tokens of a chunk
template <int LD, int ND4, int MODE>
__global__ void __launch_bounds__(OS_THREADS + 32 * OS_FEED) outer_scan_kernel(OuterScanArgs a, int tc) {
    pdl_launch_dependents();
    constexpr int DP = 4 * LD * ND4;                   // padded key size
    constexpr int TV = 2 * (OS_THREADS / LD);          // columns of a block
    constexpr bool DECAYS = OuterTraits<MODE>::DECAYS, BONUS = OuterTraits<MODE>::BONUS, GATES = OuterTraits<MODE>::GATES;
    constexpr int NVEC = DECAYS ? 3 : 2;               // vectors staged per token: r, k (and decays)
    extern __shared__ __align__(16) float os_smem[];
    // a stage: r k (w) | v | factors: wkv r . (u k), mlstm (decay, input) pairs and e^(-m)
    const int stage_floats = tc * (NVEC * DP + TV) + 4 * ((3 * tc + 3) / 4);
    const int D = a.D, Dv = a.Dv;
    const int cols = GATES ? Dv + 1 : Dv;
    const int tiles = (cols + TV - 1) / TV;
    const int h = blockIdx.x / tiles, tile = blockIdx.x - h * tiles;
    const int b = blockIdx.y;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const int j0 = tile * TV, n_cols = min(TV, cols - j0);
    const int t0 = a.cu_seqlens[b], n_b = a.cu_seqlens[b + 1] - t0;
    const int slot = a.slots[b];
    const int n_chunks = (n_b + tc - 1) / tc;
    if (n_b <= 0) { pdl_wait(); return; }

    if (warp >= OS_THREADS / 32) {
        // ---- the feeding warps: each takes every OS_FEED-th token of a chunk, the first the gates too ----------------------------------------------------------------------
        // (a row of a tensor may start anywhere: 16-byte copies only where all of them start on 16 bytes)
        const bool vec = (D & 3) == 0 &&
                         ((a.r_width | a.k_width | a.w_width | (long long)(a.r_off | a.k_off | a.w_off)) & 3) == 0 &&
                         (((uintptr_t)a.r | (uintptr_t)a.k | (uintptr_t)a.w) & 15) == 0;
        const bool vec_v = (Dv & 3) == 0 && ((a.v_width | (long long)a.v_off) & 3) == 0 && ((uintptr_t)a.v & 15) == 0;
        const int fw = warp - OS_THREADS / 32;
        if (DP > D && fw == 0) {                       // the copies never touch the padding
            const int pad = DP - D;
            for (int i = lane; i < OS_STAGES * tc * NVEC * pad; i += 32) {
                const int row = i / pad, d = D + i - row * pad;
                const int st = row / (tc * NVEC), rr = row - st * tc * NVEC;
                os_smem[st * stage_floats + rr * DP + d] = 0.0f;
            }
        }
        float ib = 0.f, fb = 0.f;
        if (GATES) { ib = a.i_bias[h]; fb = a.f_bias[h]; }
        pdl_wait();
        float m_run = 0.f;
        if (GATES) m_run = a.maxima[((size_t)slot * a.heads + h) * cols + j0];
        float raw_i[3] = {0.f, 0.f, 0.f}, raw_f[3] = {0.f, 0.f, 0.f};   // raw gates: this chunk's, the next two's
        float bonus[DP / 32];                          // (wkv) this lane's share of the head's bonus
        if (BONUS) {
#pragma unroll
            for (int e = 0; e < DP / 32; ++e) bonus[e] = lane + 32 * e < D ? a.u[h * D + lane + 32 * e] : 0.f;
        }
        const int v_cols = min(n_cols, Dv - j0);       // columns of the tile that have values (may be 0)
        auto fetch = [&](int chunk) {
            const int c0 = chunk * tc, nc = min(tc, n_b - c0);
            float* r_s = os_smem + (chunk % OS_STAGES) * stage_floats;
            float* k_s = r_s + tc * DP;
            float* w_s = k_s + tc * DP;                // (wkv)
            float* v_s = r_s + tc * NVEC * DP;
            const size_t t = (size_t)(t0 + c0);
            const float* rg = a.r + t * a.r_width + a.r_off + h * D;
            const float* kg = a.k + t * a.k_width + a.k_off + h * D;
            const float* wg = DECAYS ? a.w + t * a.w_width + a.w_off + h * D : nullptr;
            const float* vg = a.v + t * a.v_width + a.v_off + (size_t)h * Dv + j0;
            r_s += fw * DP; k_s += fw * DP; w_s += fw * DP;
            rg += fw * a.r_width; kg += fw * a.k_width; if (DECAYS) wg += fw * a.w_width;
            for (int tt = fw; tt < nc; tt += OS_FEED) {
                if (vec) {
                    for (int d = 4 * lane; d < D; d += 128) {
                        os_cp16(r_s + d, rg + d);
                        os_cp16(k_s + d, kg + d);
                        if (DECAYS) os_cp16(w_s + d, wg + d);
                    }
                } else {
                    for (int d = lane; d < D; d += 32) {
                        os_cp4(r_s + d, rg + d);
                        os_cp4(k_s + d, kg + d);
                        if (DECAYS) os_cp4(w_s + d, wg + d);
                    }
                }
                r_s += OS_FEED * DP; k_s += OS_FEED * DP; w_s += OS_FEED * DP;
                rg += OS_FEED * a.r_width; kg += OS_FEED * a.k_width; if (DECAYS) wg += OS_FEED * a.w_width;
            }
            if (vec_v && (v_cols & 3) == 0) {
                const int per = v_cols >> 2;
                for (int i = 32 * fw + lane; i < nc * per; i += 32 * OS_FEED) {
                    const int tt = i / per, cc = (i - tt * per) << 2;
                    os_cp16(v_s + tt * TV + cc, vg + (size_t)tt * a.v_width + cc);
                }
            } else {
                for (int i = 32 * fw + lane; i < nc * v_cols; i += 32 * OS_FEED) {
                    const int tt = i / v_cols, cc = i - tt * v_cols;
                    os_cp4(v_s + tt * TV + cc, vg + (size_t)tt * a.v_width + cc);
                }
            }
            if (GATES && fw == 0) {
                if (j0 + n_cols == cols)               // the normalizer's column
                    for (int tt = lane; tt < nc; tt += 32) v_s[tt * TV + n_cols - 1] = 1.0f;
                raw_i[0] = raw_i[1]; raw_f[0] = raw_f[1];
                raw_i[1] = raw_i[2]; raw_f[1] = raw_f[2];
                if (lane < nc) {
                    const float* g = a.gates + (t + lane) * a.gate_width + h;
                    raw_i[2] = g[a.i_off];
                    raw_f[2] = g[a.f_off];
                }
            }
        };
        // two chunks ahead; a chunk that does not exist is an empty group of copies
        for (int ahead = 0; ahead < 2; ++ahead) {
            if (ahead < n_chunks) fetch(ahead);
            else if (GATES) { raw_i[0] = raw_i[1]; raw_f[0] = raw_f[1]; raw_i[1] = raw_i[2]; raw_f[1] = raw_f[2]; }
            asm volatile("cp.async.commit_group;" ::: "memory");
        }
        for (int chunk = 0; chunk < n_chunks; ++chunk) {
            const int nc = min(tc, n_b - chunk * tc);
            if (chunk + 2 < n_chunks) {
                if (chunk + 2 >= OS_STAGES) os_bar_sync(OS_EMPTY((chunk + 2) % OS_STAGES));
                fetch(chunk + 2);
            } else if (GATES) {
                raw_i[0] = raw_i[1]; raw_f[0] = raw_f[1];
                raw_i[1] = raw_i[2]; raw_f[1] = raw_f[2];
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
            asm volatile("cp.async.wait_group 2;" ::: "memory");
            __syncwarp();                              // every lane's copies of this chunk are there
            float* r_s = os_smem + (chunk % OS_STAGES) * stage_floats;
            float* k_s = r_s + tc * DP;
            float* f_s = r_s + tc * (NVEC * DP + TV);
            if (BONUS) {
                // r . (u k), of the tokens this warp copied: what the current token's own value is
                // multiplied by
                constexpr int OWN = OS_TC / OS_FEED;
                float s[OWN];
#pragma unroll
                for (int i = 0; i < OWN; ++i) s[i] = 0.f;
#pragma unroll
                for (int e = 0; e < DP / 32; ++e) {
                    const int d = lane + 32 * e;
                    if (d < D) {
#pragma unroll
                        for (int i = 0; i < OWN; ++i) {
                            const int tt = fw + OS_FEED * i;
                            if (tt < nc) s[i] = fmaf(r_s[tt * DP + d] * bonus[e], k_s[tt * DP + d], s[i]);
                        }
                    }
                }
#pragma unroll
                for (int o = 16; o > 0; o >>= 1) {
#pragma unroll
                    for (int i = 0; i < OWN; ++i) s[i] += __shfl_xor_sync(0xffffffffu, s[i], o);
                }
                if (lane == 0) {
#pragma unroll
                    for (int i = 0; i < OWN; ++i)
                        if (fw + OS_FEED * i < nc) f_s[fw + OS_FEED * i] = s[i];
                }
            } else if (GATES && fw == 0) {
                // a token a lane; the maxima by a scan in which a stretch of tokens is the pair
                // (sum of f, largest i + the f's after it)
                const bool mine = lane < nc;
                const float li = mine ? os_soft_cap(raw_i[0] + ib, a.cap) : -INFINITY;
                const float zf = mine ? os_soft_cap(raw_f[0] + fb, a.cap) : 0.f;
                const float lf = mine ? fminf(zf, 0.f) - log1pf(expf(-fabsf(zf))) : 0.f;
                float F = lf, M = li;
#pragma unroll
                for (int o = 1; o < OS_TC; o <<= 1) {
                    const float pF = __shfl_up_sync(0xffffffffu, F, o), pM = __shfl_up_sync(0xffffffffu, M, o);
                    if (lane >= o) { M = fmaxf(pM + F, M); F = pF + F; }
                }
                const float m_t = fmaxf(F + m_run, M);
                float before = __shfl_up_sync(0xffffffffu, m_t, 1);
                if (lane == 0) before = m_run;
                if (mine) {
                    // (m_t is often lf + before, rounded: in this order the difference is exact, so what m_t
                    // lost in rounding stays in the state's factor instead of adding up token by token)
                    f_s[2 * lane] = expf((before - m_t) + lf);
                    f_s[2 * lane + 1] = expf(li - m_t);
                    f_s[2 * tc + lane] = expf(-m_t);
                }
                m_run = __shfl_sync(0xffffffffu, m_t, nc - 1);
            }
            os_bar_arrive(OS_FULL(chunk % OS_STAGES));
        }
        if (GATES && fw == 0)
            for (int i = lane; i < n_cols; i += 32) a.maxima[((size_t)slot * a.heads + h) * cols + j0 + i] = m_run;
        return;
    }

    // ---- the four warps that walk the tokens ---------------------------------------------------------
    const int l = tid % LD, c = tid / LD;              // lane of the pair's group; pair of columns
    const bool live0 = 2 * c < n_cols, live1 = 2 * c + 1 < n_cols;
    pdl_wait();
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
    const size_t out_row = (size_t)a.heads * Dv;
    float* out0 = a.out + (size_t)t0 * out_row + (size_t)h * Dv + j0;
    // number `x` is the sum of token t (of the chunk, whose first token's output row is o) and column cc
    auto emit = [&](float x, float* o, const float* v_s, const float* f_s, int t, int cc, int token) {
        if (cc >= n_cols) return;
        if (BONUS) o[t * out_row + cc] = fmaf(f_s[t], v_s[t * TV + cc], x);
        else if (j0 + cc < Dv) o[t * out_row + cc] = x * a.r_scale;
        else a.den[(size_t)(token + t) * a.heads + h] = fmaxf(fabsf(x * a.r_scale), f_s[2 * tc + t]) + 1e-6f;
    };
    for (int chunk = 0; chunk < n_chunks; ++chunk) {
        const int stage = chunk % OS_STAGES;
        const int nc = min(tc, n_b - chunk * tc);
        os_bar_sync(OS_FULL(stage));
        const float* r_s = os_smem + stage * stage_floats;
        const float* v_s = r_s + tc * NVEC * DP;
        const float* f_s = v_s + tc * TV;
        const float4* r4 = reinterpret_cast<const float4*>(r_s) + l;
        const float4* k4 = r4 + tc * (DP / 4);
        const float4* w4 = k4 + tc * (DP / 4);
        float* o = out0 + (size_t)chunk * tc * out_row;
        const int token = t0 + chunk * tc;
        int tt = 0;
        for (; tt + OS_TU <= nc; tt += OS_TU) {
            float acc[2 * OS_TU];
#pragma unroll
            for (int u = 0; u < OS_TU; ++u) {
                const int t = tt + u;
                float2 vv = *reinterpret_cast<const float2*>(v_s + t * TV + 2 * c);
                float keep = 0.f;
                if (GATES) {
                    const float2 f = *reinterpret_cast<const float2*>(f_s + 2 * t);
                    keep = f.x; vv.x *= f.y; vv.y *= f.y;
                }
                os_token<ND4, MODE>(S0, S1, r4 + t * (DP / 4), k4 + t * (DP / 4), w4 + t * (DP / 4), keep, vv.x, vv.y, LD,
                                   acc[2 * u], acc[2 * u + 1]);
            }
            os_reduce16<LD>(acc, l);
            if (LD == 8) {
                emit(acc[0], o, v_s, f_s, tt + l, 2 * c, token);
                emit(acc[1], o, v_s, f_s, tt + l, 2 * c + 1, token);
            } else if (LD == 16) {
                emit(acc[0], o, v_s, f_s, tt + (l >> 1), 2 * c + (l & 1), token);
            } else if ((l & 1) == 0) {
                emit(acc[0], o, v_s, f_s, tt + (l >> 2), 2 * c + ((l >> 1) & 1), token);
            }
        }
        for (; tt < nc; ++tt) {
            float2 vv = *reinterpret_cast<const float2*>(v_s + tt * TV + 2 * c);
            float keep = 0.f, a0, a1;
            if (GATES) {
                const float2 f = *reinterpret_cast<const float2*>(f_s + 2 * tt);
                keep = f.x; vv.x *= f.y; vv.y *= f.y;
            }
            os_token<ND4, MODE>(S0, S1, r4 + tt * (DP / 4), k4 + tt * (DP / 4), w4 + tt * (DP / 4), keep, vv.x, vv.y, LD, a0, a1);
#pragma unroll
            for (int o2 = LD / 2; o2 > 0; o2 >>= 1) {
                a0 += __shfl_xor_sync(0xffffffffu, a0, o2);
                a1 += __shfl_xor_sync(0xffffffffu, a1, o2);
            }
            if (l == 0) {
                emit(a0, o, v_s, f_s, tt, 2 * c, token);
                emit(a1, o, v_s, f_s, tt, 2 * c + 1, token);
            }
        }
        // (only a stage that will be filled again is handed back: nobody waits for the others)
        if (chunk + OS_STAGES < n_chunks) os_bar_arrive(OS_EMPTY(stage));
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
}

template <int LD, int ND4, int MODE>
static int os_launch(const OuterScanArgs& a, int max_tokens, cudaStream_t stream) {
    constexpr int DP = 4 * LD * ND4, TV = 2 * (OS_THREADS / LD), NVEC = OuterTraits<MODE>::DECAYS ? 3 : 2;
    // (short rows take shorter chunks, so that more blocks fit an SM: single tokens most of all)
    const int tc = max_tokens < 1 ? OS_TC : max_tokens < OS_TC ? max_tokens : OS_TC;
    auto bytes = [&](int t) { return (size_t)OS_STAGES * (t * (NVEC * DP + TV) + 4 * ((3 * t + 3) / 4)) * sizeof(float); };
    static bool configured[64] = {false};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return MF_ERR_UNSUPPORTED;
    if (!configured[dev]) {
        cudaError_t e = cudaFuncSetAttribute(outer_scan_kernel<LD, ND4, MODE>,
                                             cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes(OS_TC));
        if (e != cudaSuccess) return (int)e;
        configured[dev] = true;
    }
    const int cols = OuterTraits<MODE>::GATES ? a.Dv + 1 : a.Dv;
    const int tiles = (cols + TV - 1) / TV;
    mf_launch(outer_scan_kernel<LD, ND4, MODE>, dim3(a.heads * tiles, a.n_rows), dim3(OS_THREADS + 32 * OS_FEED), bytes(tc),
              stream, a, tc);
    return MF_LAUNCH_CHECK();
}

template <int MODE>
static int os_choose(const OuterScanArgs& a, int max_tokens, cudaStream_t stream) {
    if (a.n_rows <= 0) return 0;
    if (a.D < 1 || a.D > OS_MAX_D || a.Dv < 1 || a.heads < 1 || a.n_rows > 65535) return MF_ERR_UNSUPPORTED;
    if (((uintptr_t)a.state & 15) != 0) return MF_ERR_UNSUPPORTED;
    if (a.D <= 32) return os_launch<8, 1, MODE>(a, max_tokens, stream);
    if (a.D <= 64) return os_launch<16, 1, MODE>(a, max_tokens, stream);
    if (a.D <= 128) return os_launch<16, 2, MODE>(a, max_tokens, stream);
    return os_launch<32, 2, MODE>(a, max_tokens, stream);
}

// max_tokens: the most tokens a row brings (0: not known; it only sizes the chunks)
extern "C" int mf_wkv_scan(const OuterScanArgs* args, int max_tokens, cudaStream_t stream) {
    return os_choose<OS_WKV>(*args, max_tokens, stream);
}
extern "C" int mf_mlstm_scan(const OuterScanArgs* args, int max_tokens, cudaStream_t stream) {
    if (!(args->cap > 0.0f)) return MF_ERR_ARGUMENT;
    return os_choose<OS_MLSTM>(*args, max_tokens, stream);
}
extern "C" int mf_gla_scan(const OuterScanArgs* args, int max_tokens, cudaStream_t stream) {
    return os_choose<OS_GLA>(*args, max_tokens, stream);
}

// ------------------------------------------------------------------------------------------
// out[t][c] = exp(-exp(w0[c] + sum_r w2t[r][c] tanh(t1[t][r]))) or, SIGMOID, with z = w0[c] + sum_r
// w2t[r][c] t1[t][r], sigmoid(z)^inv_tau = exp(inv_tau log sigmoid(z)): a thread per channel, WD_T
// tokens a block, whose tanh(t1) (t1) lie in shared memory.
// ------------------------------------------------------------------------------------------
#define WD_T 16

template <int NT, bool SIGMOID>
__global__ void __launch_bounds__(128)
low_rank_decay_kernel(const float* __restrict__ t1, long long t1_width, const float* __restrict__ w2t,
                 const float* __restrict__ w0, float* __restrict__ out, int n_tokens, int rank, int channels,
                      float inv_tau) {
    pdl_prologue();
    extern __shared__ __align__(16) float wd_s[];      // [NT][rank, padded to a multiple of 4]
    const int first = blockIdx.y * NT, nt = min(NT, n_tokens - first);
    const int pitch = (rank + 3) & ~3;
    for (int i = threadIdx.x; i < NT * rank; i += blockDim.x) {
        const int t = i / rank, r = i - t * rank;
        const float x = t < nt ? t1[(size_t)(first + t) * t1_width + r] : 0.f;
        wd_s[t * pitch + r] = SIGMOID ? x : tanhf(x);
    }
    __syncthreads();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    float acc[NT];
    const float base = w0[c];
#pragma unroll
    for (int t = 0; t < NT; ++t) acc[t] = base;
    int r = 0;
    // four numbers of the rank at a time (every row of wd_s starts on 16 bytes); few tokens: more of the
    // matrix's loads in flight, since nothing else hides them
    constexpr int AHEAD = NT <= 2 ? 4 : 2;
    for (; r + 4 * AHEAD <= rank; r += 4 * AHEAD) {
        float w[4 * AHEAD];
#pragma unroll
        for (int i = 0; i < 4 * AHEAD; ++i) w[i] = w2t[(size_t)(r + i) * channels + c];
#pragma unroll
        for (int t = 0; t < NT; ++t) {
#pragma unroll
            for (int i = 0; i < AHEAD; ++i) {
                const float4 x = *reinterpret_cast<const float4*>(wd_s + t * pitch + r + 4 * i);
                acc[t] = fmaf(w[4 * i], x.x, acc[t]);
                acc[t] = fmaf(w[4 * i + 1], x.y, acc[t]);
                acc[t] = fmaf(w[4 * i + 2], x.z, acc[t]);
                acc[t] = fmaf(w[4 * i + 3], x.w, acc[t]);
            }
        }
    }
    for (; r < rank; ++r) {
        const float w = w2t[(size_t)r * channels + c];
#pragma unroll
        for (int t = 0; t < NT; ++t) acc[t] = fmaf(w, wd_s[t * pitch + r], acc[t]);
    }
#pragma unroll
    for (int t = 0; t < NT; ++t)
        if (t < nt)
            out[(size_t)(first + t) * channels + c] =
                SIGMOID ? expf(inv_tau * (fminf(acc[t], 0.f) - log1pf(expf(-fabsf(acc[t]))))) : expf(-expf(acc[t]));
}

template <bool SIGMOID>
static int low_rank_decay(const float* t1, long long t1_width, const float* w2t, const float* w0, float* out,
                          int n_tokens, int rank, int channels, float inv_tau, cudaStream_t stream) {
    if (n_tokens <= 0) return 0;
    if (rank < 1 || channels < 1 || (size_t)(rank + 3) * WD_T * sizeof(float) > 48 * 1024) return MF_ERR_UNSUPPORTED;
    const int cb = (channels + 127) / 128;
    if (n_tokens <= 64) {
        if ((n_tokens + 1) / 2 > 65535) return MF_ERR_UNSUPPORTED;
        mf_launch(low_rank_decay_kernel<2, SIGMOID>, dim3(cb, (n_tokens + 1) / 2), dim3(128), (size_t)((rank + 3) & ~3) * 2 * sizeof(float),
                  stream, t1, t1_width, w2t, w0, out, n_tokens, rank, channels, inv_tau);
    } else {
        if ((n_tokens + WD_T - 1) / WD_T > 65535) return MF_ERR_UNSUPPORTED;
        mf_launch(low_rank_decay_kernel<WD_T, SIGMOID>, dim3(cb, (n_tokens + WD_T - 1) / WD_T), dim3(128),
                  (size_t)((rank + 3) & ~3) * WD_T * sizeof(float), stream, t1, t1_width, w2t, w0, out, n_tokens, rank, channels, inv_tau);
    }
    return MF_LAUNCH_CHECK();
}

extern "C" int mf_wkv_decay(const float* t1, long long t1_width, const float* w2t, const float* w0,
                            float* out, int n_tokens, int rank, int channels, cudaStream_t stream) {
    return low_rank_decay<false>(t1, t1_width, w2t, w0, out, n_tokens, rank, channels, 1.0f, stream);
}
extern "C" int mf_sigmoid_decay(const float* t1, long long t1_width, const float* w2t, const float* w0, float* out,
                                int n_tokens, int rank, int channels, float inv_tau, cudaStream_t stream) {
    return low_rank_decay<true>(t1, t1_width, w2t, w0, out, n_tokens, rank, channels, inv_tau, stream);
}
