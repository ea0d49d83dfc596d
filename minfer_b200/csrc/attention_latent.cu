// Attention of single queries over one wide latent vector per position that serves as key and value
// of all heads (bfloat16, vectors of up to 640 numbers): what the kernels for single queries whose
// warps each own a tile of keys cannot hold, since a warp's output sums would fill its registers.
//
// Every row of q is a query at its own position with all its heads; up to 16 heads are the 16 rows of
// an m16n8k16 MMA, so a latent vector is read once for all of them.  Keys are walked a page (64
// positions) at a time through two cp.async buffers; rows are padded by 16 bytes, which keeps
// ldmatrix free of bank conflicts.  The eight warps of a block share a page:
//   scores     a warp takes 8 keys over the whole width
//   softmax    a warp takes two of the 16 rows: running maximum and sum in float32, base 2
//   values     a warp takes every eighth stretch of 16 output columns over all 64 keys
// The first `vd` numbers of a vector are the value.  Few queries over many keys: the pages are dealt
// to several blocks, whose results latent_combine merges in order.  The sink (a key without a value)
// is added once, at the end.
#include "common.cuh"

#define LA_WARPS 8
#define LA_HEADS 16
#define LA_MAX_W 640

struct LatentArgs {
    const __nv_bfloat16* q;   // [rows][n_heads][kw]
    const __nv_bfloat16* k;   // cache [pages][1][64][kw]
    const int* row_seq;       // [rows] batch row of each query
    const int* row_pos;       // [rows] absolute position of each query
    const int* page_table;
    int table_stride, ring;
    __nv_bfloat16* out;       // [rows][n_heads * vd]
    float* partial;           // [rows][n_heads][n_splits][vd + 2]   (n_splits > 1)
    const float* sink_logit;  // [n_heads] or null for 0
    int n_heads, kw, vd, window, sink, tiles_per_cta, n_splits;
    float scale_log2;
};

__device__ __forceinline__ void la_mma(float* d, const uint32_t* a, uint32_t b0, uint32_t b1) {
    asm volatile(
        "mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9},"
        " {%0, %1, %2, %3};"
        : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
        : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void la_ldsm(uint32_t addr, uint32_t* r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ void la_ldsm_trans(uint32_t addr, uint32_t* r) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}

__host__ __device__ constexpr int la_pitch(int kw) { return ((kw + 15) / 16) * 32 + 16; }   // bytes of a row
#define LA_SP 68              // floats of a row of scores
#define LA_PP 144             // bytes of a row of weights
static size_t la_smem(int kw) {
    return (size_t)(2 * MF_PAGE + LA_HEADS) * la_pitch(kw) + LA_HEADS * LA_SP * 4 + LA_HEADS * LA_PP + 3 * LA_HEADS * 4;
}

// NP: stretches of 16 output columns a warp takes (vd <= 128 NP)
template <int NP>
__global__ void __launch_bounds__(LA_WARPS * 32) latent_decode_kernel(LatentArgs a) {
    pdl_launch_dependents();
    extern __shared__ __align__(128) uint8_t la_buf[];
    const int pitch = la_pitch(a.kw), kp = ((a.kw + 15) / 16) * 16;
    uint8_t* q_b = la_buf + 2 * MF_PAGE * pitch;
    float* s_s = reinterpret_cast<float*>(q_b + LA_HEADS * pitch);
    uint8_t* p_b = reinterpret_cast<uint8_t*>(s_s + LA_HEADS * LA_SP);
    float* corr_s = reinterpret_cast<float*>(p_b + LA_HEADS * LA_PP);
    float* m_s = corr_s + LA_HEADS;
    float* l_s = m_s + LA_HEADS;
    const uint32_t k_base = (uint32_t)__cvta_generic_to_shared(la_buf);
    const uint32_t q_base = (uint32_t)__cvta_generic_to_shared(q_b);
    const uint32_t p_base = (uint32_t)__cvta_generic_to_shared(p_b);
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, g = lane >> 2, t = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * LA_HEADS, row = blockIdx.z;
    const int n_h = min(LA_HEADS, a.n_heads - h0);
    const int b = a.row_seq[row], pos = a.row_pos[row];
    const int lo = a.window > 0 ? max(0, pos - a.window + 1) : 0;
    const int tile_lo = lo / MF_PAGE + split * a.tiles_per_cta;
    const int tile_hi = min(pos / MF_PAGE, tile_lo + a.tiles_per_cta - 1);     // inclusive
    // columns kw .. kp of keys and queries stay zero: no copy touches them
    for (int i = tid; i < (2 * MF_PAGE + LA_HEADS) * (kp - a.kw); i += LA_WARPS * 32) {
        const int r = i / (kp - a.kw), c = a.kw + i - r * (kp - a.kw);
        *reinterpret_cast<__nv_bfloat16*>(la_buf + (size_t)r * pitch + 2 * c) = __float2bfloat16_rn(0.f);
    }
    pdl_wait();
    const int chunks = a.kw >> 3;                     // 16-byte pieces of a vector
    auto load_tile = [&](int tile, int buf) {
        const int key0 = tile * MF_PAGE, p_eff = a.ring > 0 ? key0 % a.ring : key0;
        int page = a.page_table[(size_t)b * a.table_stride + (p_eff >> 6)];
        if (page < 0) page = 0;                       // (masked: no visible position lies there)
        const __nv_bfloat16* src = a.k + (size_t)page * MF_PAGE * a.kw;
        const uint32_t dst = k_base + (uint32_t)(buf * MF_PAGE * pitch);
#pragma unroll
        for (int i = 0; i < MF_PAGE / LA_WARPS; ++i) {
            const int r = warp + LA_WARPS * i;
            for (int c = lane; c < chunks; c += 32)
                asm volatile("cp.async.cg.shared.global [%0], [%1], 16;"
                             ::"r"(dst + (uint32_t)(r * pitch + c * 16)), "l"(src + (size_t)r * a.kw + c * 8) : "memory");
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    if (tile_lo <= tile_hi) load_tile(tile_lo, 0);
    for (int i = tid; i < LA_HEADS * chunks; i += LA_WARPS * 32) {
        const int r = i / chunks, c = i - r * chunks;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < n_h) v = *reinterpret_cast<const uint4*>(a.q + ((size_t)row * a.n_heads + h0 + r) * a.kw + c * 8);
        *reinterpret_cast<uint4*>(q_b + r * pitch + c * 16) = v;
    }
    // this warp's two rows of the softmax
    float m_r[2] = {-INFINITY, -INFINITY}, l_r[2] = {0.f, 0.f};
    float o[NP][2][4];
#pragma unroll
    for (int i = 0; i < NP; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) o[i][j][0] = o[i][j][1] = o[i][j][2] = o[i][j][3] = 0.f;
    const uint32_t a_lane = (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 16);
    const uint32_t b_lane = (uint32_t)((8 * warp + (lane & 7)) * pitch + (lane >> 3) * 16);
    const uint32_t b_lane_last = (uint32_t)((8 * warp + (lane & 7)) * pitch + ((lane >> 3) & 1) * 16);
    const uint32_t v_lane = (uint32_t)((((lane >> 3) & 1) * 8 + (lane & 7)) * pitch + (lane >> 4) * 16);
    const uint32_t p_lane = (uint32_t)(((lane & 7) + ((lane >> 3) & 1) * 8) * LA_PP + (lane >> 4) * 16);
    const int ksteps = kp >> 4;
    const int n_pairs = (a.vd + 15) >> 4;

    for (int tile = tile_lo, buf = 0; tile <= tile_hi; ++tile, buf ^= 1) {
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                              // the page is here, the one before is read
        if (tile < tile_hi) load_tile(tile + 1, buf ^ 1);
        const uint32_t ks_base = k_base + (uint32_t)(buf * MF_PAGE * pitch);
        // ---- scores of this warp's 8 keys
        float s0[4] = {0.f, 0.f, 0.f, 0.f}, s1[4] = {0.f, 0.f, 0.f, 0.f};
        int ks = 0;
#pragma unroll 2
        for (; ks + 2 <= ksteps; ks += 2) {
            uint32_t qa[4], qb[4], kb[4];
            la_ldsm(q_base + a_lane + (uint32_t)(ks * 32), qa);
            la_ldsm(q_base + a_lane + (uint32_t)(ks * 32 + 32), qb);
            la_ldsm(ks_base + b_lane + (uint32_t)(ks * 32), kb);
            la_mma(s0, qa, kb[0], kb[1]);
            la_mma(s1, qb, kb[2], kb[3]);
        }
        if (ks < ksteps) {
            uint32_t qa[4], kb[4];
            la_ldsm(q_base + a_lane + (uint32_t)(ks * 32), qa);
            la_ldsm(ks_base + b_lane_last + (uint32_t)(ks * 32), kb);
            la_mma(s0, qa, kb[0], kb[1]);
        }
        float* sr = s_s + g * LA_SP + 8 * warp + 2 * t;
        sr[0] = s0[0] + s1[0]; sr[1] = s0[1] + s1[1];
        sr[8 * LA_SP] = s0[2] + s1[2]; sr[8 * LA_SP + 1] = s0[3] + s1[3];
        __syncthreads();
        // ---- softmax of this warp's two rows
#pragma unroll
        for (int r = 0; r < 2; ++r) {
            const int hr = 2 * warp + r;
            float x[2];
#pragma unroll
            for (int j = 0; j < 2; ++j) {
                const int key = tile * MF_PAGE + lane + 32 * j;
                const bool vis = key <= pos && key >= lo;
                x[j] = vis ? s_s[hr * LA_SP + lane + 32 * j] * a.scale_log2 : -INFINITY;
            }
            const float m_new = fmaxf(m_r[r], warp_max(fmaxf(x[0], x[1])));
            const float m_use = m_new == -INFINITY ? 0.f : m_new;
            const float corr = m_r[r] == -INFINITY ? 0.f : exp2f(m_r[r] - m_use);
            const float p0 = exp2f(x[0] - m_use), p1 = exp2f(x[1] - m_use);
            m_r[r] = m_new;
            l_r[r] = l_r[r] * corr + warp_sum(p0 + p1);
            __nv_bfloat16* pr = reinterpret_cast<__nv_bfloat16*>(p_b + hr * LA_PP);
            pr[lane] = __float2bfloat16_rn(p0);
            pr[lane + 32] = __float2bfloat16_rn(p1);
            if (lane == 0) corr_s[hr] = corr;
        }
        __syncthreads();
        // ---- values: this warp's output columns over the page's 64 keys
        const float c0 = corr_s[g], c1 = corr_s[g + 8];
        uint32_t pa[4][4];
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) la_ldsm(p_base + p_lane + (uint32_t)(kk * 32), pa[kk]);
#pragma unroll
        for (int i = 0; i < NP; ++i) {
            const int pair = warp + LA_WARPS * i;
            if (pair < n_pairs) {
#pragma unroll
                for (int j = 0; j < 2; ++j) { o[i][j][0] *= c0; o[i][j][1] *= c0; o[i][j][2] *= c1; o[i][j][3] *= c1; }
#pragma unroll
                for (int kk = 0; kk < 4; ++kk) {
                    uint32_t v[4];
                    la_ldsm_trans(ks_base + v_lane + (uint32_t)(kk * 16 * pitch + pair * 32), v);
                    la_mma(o[i][0], pa[kk], v[0], v[1]);
                    la_mma(o[i][1], pa[kk], v[2], v[3]);
                }
            }
        }
    }
    if (lane == 0) {
#pragma unroll
        for (int r = 0; r < 2; ++r) { m_s[2 * warp + r] = m_r[r]; l_s[2 * warp + r] = l_r[r]; }
    }
    __syncthreads();
    // rows g and g + 8 of the product are heads h0 + g and h0 + g + 8
#pragma unroll
    for (int r = 0; r < 2; ++r) {
        const int hr = g + 8 * r;
        if (hr >= n_h) continue;
        const int head = h0 + hr;
        const float m = m_s[hr], l = l_s[hr];
        if (a.n_splits > 1) {
            float* part = a.partial + (((size_t)row * a.n_heads + head) * a.n_splits + split) * (a.vd + 2);
            if (warp == 0 && t == 0) { part[0] = m; part[1] = l; }
#pragma unroll
            for (int i = 0; i < NP; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int c = (warp + LA_WARPS * i) * 16 + 8 * j + 2 * t;
                    if (c < a.vd) { part[2 + c] = o[i][j][2 * r]; part[3 + c] = o[i][j][2 * r + 1]; }
                }
        } else {
            float f = 1.0f / l;
            if (a.sink) {
                const float sink2 = a.sink_logit ? a.sink_logit[head] * 1.4426950408889634f : 0.f;
                const float mf = fmaxf(m, sink2);
                const float e = exp2f(m - mf);
                f = e / (l * e + exp2f(sink2 - mf));
            }
#pragma unroll
            for (int i = 0; i < NP; ++i)
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    const int c = (warp + LA_WARPS * i) * 16 + 8 * j + 2 * t;
                    if (c < a.vd)
                        *reinterpret_cast<__nv_bfloat162*>(a.out + ((size_t)row * a.n_heads + head) * a.vd + c) =
                            __floats2bfloat162_rn(o[i][j][2 * r] * f, o[i][j][2 * r + 1] * f);
                }
        }
    }
}

// Merges the splits of one (query, head) in split order and adds the sink.  The splits' factors are
// formed once, then every output number is a sum of independent loads.
#define LA_MAX_SPLITS 512
__global__ void __launch_bounds__(256)
latent_combine_kernel(const float* __restrict__ partial, __nv_bfloat16* __restrict__ out, int n_splits, int vd,
                      int sink, const float* __restrict__ sink_logit, int n_heads) {
    pdl_prologue();
    __shared__ float f_s[LA_MAX_SPLITS];
    __shared__ float scratch[33];
    const size_t rh = blockIdx.x, stride = (size_t)(vd + 2);
    const float* p = partial + rh * n_splits * stride;
    const float sink2 = (sink && sink_logit) ? sink_logit[rh % n_heads] * 1.4426950408889634f : 0.f;
    float m = sink ? sink2 : -INFINITY;
    for (int c = threadIdx.x; c < n_splits; c += blockDim.x) m = fmaxf(m, p[c * stride]);
    m = block_max(m, scratch);
    float l = 0.f;
    for (int c = threadIdx.x; c < n_splits; c += blockDim.x) {
        const float2 ml = *reinterpret_cast<const float2*>(p + c * stride);
        const float f = exp2f(ml.x - m);               // (a split that saw nothing has maximum -inf: 0)
        f_s[c] = f;
        l = fmaf(ml.y, f, l);
    }
    l = block_sum(l, scratch);                         // (its barriers also publish f_s)
    if (sink) l += exp2f(sink2 - m);
    const float inv = 1.0f / l;
    for (int d = 2 * threadIdx.x; d < vd; d += 2 * blockDim.x) {
        const float* pd = p + 2 + d;
        float2 acc = make_float2(0.f, 0.f);
#pragma unroll 16
        for (int c = 0; c < n_splits; ++c) {
            const float2 x = *reinterpret_cast<const float2*>(pd + c * stride);
            acc.x = fmaf(x.x, f_s[c], acc.x);
            acc.y = fmaf(x.y, f_s[c], acc.y);
        }
        *reinterpret_cast<__nv_bfloat162*>(out + rh * vd + d) = __floats2bfloat162_rn(acc.x * inv, acc.y * inv);
    }
}

extern "C" int mf_latent_supported(int kw, int vd) {
    return kw >= 8 && kw <= LA_MAX_W && kw % 8 == 0 && vd >= 8 && vd <= kw && vd % 8 == 0;
}

// How the pages of single queries are dealt: pages a block, splits; from the sizes only.
// `reach_keys`: the most keys a query sees.
extern "C" int mf_latent_plan(int rows, int n_heads, int kw, int reach_keys, int* tiles_per_cta, int* n_splits) {
    const int n_tiles = (reach_keys + MF_PAGE - 1) / MF_PAGE + 1;          // the range need not start on a page
    const int blocks = rows * ((n_heads + LA_HEADS - 1) / LA_HEADS);
    int per_sm = (int)(220 * 1024 / la_smem(kw));
    if (per_sm > 3) per_sm = 3;
    if (per_sm < 1) per_sm = 1;
    int splits = blocks > 0 ? (per_sm * mf_sm_count()) / blocks : 1;
    if (splits > n_tiles) splits = n_tiles;
    if (splits > LA_MAX_SPLITS) splits = LA_MAX_SPLITS;
    if (splits < 1) splits = 1;
    const int tpc = (n_tiles + splits - 1) / splits;
    *tiles_per_cta = tpc;
    *n_splits = (n_tiles + tpc - 1) / tpc;
    return 0;
}

template <int NP>
static int la_launch(const LatentArgs& a, int rows, cudaStream_t stream) {
    const size_t smem = la_smem(a.kw);
    static bool configured[64] = {false};
    int dev = 0;
    if (cudaGetDevice(&dev) != cudaSuccess || dev < 0 || dev >= 64) return MF_ERR_UNSUPPORTED;
    if (!configured[dev]) {
        cudaError_t e = cudaFuncSetAttribute(latent_decode_kernel<NP>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (int)la_smem(LA_MAX_W));
        if (e != cudaSuccess) return (int)e;
        configured[dev] = true;
    }
    mf_launch(latent_decode_kernel<NP>, dim3(a.n_splits, (a.n_heads + LA_HEADS - 1) / LA_HEADS, rows),
              dim3(LA_WARPS * 32), smem, stream, a);
    return MF_LAUNCH_CHECK();
}

// Every row of q [rows][n_heads][kw] (bfloat16) is a query at row_pos over the paged cache of latent
// vectors; out [rows][n_heads * vd].  `partial`: rows * n_heads * splits * (vd + 2) floats when the plan
// has more than one split.
extern "C" int mf_latent_decode(const void* q, const void* k_cache, const int* row_seq, const int* row_pos,
                                const int* page_table, int table_stride, int ring, void* out, float* partial,
                                int rows, int n_heads, int kw, int vd, int window, int sink, float scale,
                                int reach_keys, const float* sink_logit, cudaStream_t stream) {
    if (rows <= 0) return 0;
    if (!mf_latent_supported(kw, vd) || n_heads < 1 || rows > 65535) return MF_ERR_UNSUPPORTED;
    if (page_table == nullptr || window < 0 || ring < 0 || ring % MF_PAGE != 0) return MF_ERR_ARGUMENT;
    if (((uintptr_t)q | (uintptr_t)k_cache) & 15 || (uintptr_t)out & 3) return MF_ERR_UNSUPPORTED;
    LatentArgs a;
    a.q = (const __nv_bfloat16*)q; a.k = (const __nv_bfloat16*)k_cache;
    a.row_seq = row_seq; a.row_pos = row_pos; a.page_table = page_table;
    a.table_stride = table_stride; a.ring = ring;
    a.out = (__nv_bfloat16*)out; a.partial = partial; a.sink_logit = sink_logit;
    a.n_heads = n_heads; a.kw = kw; a.vd = vd; a.window = window; a.sink = sink ? 1 : 0;
    a.scale_log2 = scale * 1.4426950408889634f;
    mf_latent_plan(rows, n_heads, kw, reach_keys, &a.tiles_per_cta, &a.n_splits);
    if (a.n_splits > 1 && partial == nullptr) return MF_ERR_ARGUMENT;
    int e;
    if (vd <= 128) e = la_launch<1>(a, rows, stream);
    else if (vd <= 256) e = la_launch<2>(a, rows, stream);
    else if (vd <= 384) e = la_launch<3>(a, rows, stream);
    else if (vd <= 512) e = la_launch<4>(a, rows, stream);
    else e = la_launch<5>(a, rows, stream);
    if (e || a.n_splits == 1) return e;
    mf_launch_ex(false, latent_combine_kernel, dim3(rows * n_heads), dim3(vd <= 256 ? 128 : 256), 0, stream, (const float*)partial,
                 (__nv_bfloat16*)out, a.n_splits, vd, a.sink, sink_logit, n_heads);
    return MF_LAUNCH_CHECK();
}
