// Latent attention over a paged latent cache.
//
// Keys and values of all heads are linear in a per-token latent: k[h] = [Wuk[h] c | k_rot], v[h] = Wuv[h] c, where k_rot is
// one rotated key part shared by the heads.  A token's cache entry is therefore only [c | k_rot] (rank + rot components),
// and a score can be taken without expanding the keys:
//     q[h] . k[h] = (Wuk[h]^T q_nope[h]) . c + q_rot[h] . k_rot,
// i.e. a dot product of a (rank + rot)-wide "latent query" with the cache entry; the weighted sum of the latents is
// expanded to values once per query.  That form serves decode steps and short portions of a prompt: the cache entry is
// read once for all heads.  Long portions expand keys and values instead (decoder.cu) and run the flash kernel.
//
// Kernels: latent_prep (norm of the latent, rotations, append), latent_project_* (queries into the latent space, latents to
// values: one small matrix per head), latent_attn_* (scores, softmax, weighted sum; split over the keys when there are few
// queries), latent_combine (merges the splits), latent_gather (contiguous copy of cached entries).
#include "decoder_ops.cuh"
#include "mma_utils.cuh"
#include "tc_utils.cuh"
#include <math.h>
#include <algorithm>

namespace jsm {

using tc::smem_u32;

constexpr int PAGE = JSM_PAGE_SIZE;

// ---- append and rotation ------------------------------------------------------------------------------------------
// qd row of a token: [q head 0 (qh) | ... | down: c (rank), key part (rot)].  Blocks (token, part): the last part makes the
// cache entry, the others 256 groups of 8 query components each.  vec: the boundaries between the unrotated part, the two
// halves of the rotated part and the padding are multiples of 8.
template <typename T>
__device__ __forceinline__ void store8(T* p, const float (&v)[8]);
template <>
__device__ __forceinline__ void store8<float>(float* p, const float (&v)[8]) {
    reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
    reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
}
template <>
__device__ __forceinline__ void store8<__nv_bfloat16>(__nv_bfloat16* p, const float (&v)[8]) {
    *reinterpret_cast<uint4*>(p) = make_uint4(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]), pack_bf16x2(v[4], v[5]), pack_bf16x2(v[6], v[7]));
}
__device__ __forceinline__ void load8(const float* p, float (&v)[8]) {
    const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
}

template <typename T>
__global__ void __launch_bounds__(256) latent_prep_kernel(const float* __restrict__ qd, LatentDims d, const float* __restrict__ gain, float eps,
                                                          T* __restrict__ pool, const int32_t* __restrict__ block_table, int max_pages,
                                                          const float2* __restrict__ rope, const int32_t* __restrict__ tok_row,
                                                          const int32_t* __restrict__ tok_pos, T* __restrict__ q, T* __restrict__ q_lat, int vec) {
    __shared__ float red[8];
    chain_trigger();
    chain_wait();
    const int t = blockIdx.x;
    const int qh = pad8(d.dim + d.rot), cr = pad8(d.rank + d.rot), q_cols = d.H * qh, half = d.rot / 2;
    const float* src = qd + (long long)t * (q_cols + cr);
    const int pos = tok_pos[t];
    const float2* cs = rope + (long long)pos * half;
    if (blockIdx.y + 1 < gridDim.y) {
        // queries: unrotated components copied, the rest rotated (component i with i + rot/2)
        const int i0 = (blockIdx.y * 256 + threadIdx.x) * 8;
        if (i0 >= q_cols) return;
        const int j0 = i0 % qh;
        float v[8];
        if (vec) {
            load8(src + i0, v);
            if (j0 >= d.dim + d.rot) {
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = 0.0f;
            } else if (j0 >= d.dim) {
                const int r = j0 - d.dim;
                const bool lower = r < half;
                const int p = lower ? r : r - half;
                float o[8], c[16];
                load8(src + (lower ? i0 + half : i0 - half), o);
                load8(reinterpret_cast<const float*>(cs + p), reinterpret_cast<float(&)[8]>(c[0]));
                load8(reinterpret_cast<const float*>(cs + p + 4), reinterpret_cast<float(&)[8]>(c[8]));
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = lower ? v[e] * c[2 * e] - o[e] * c[2 * e + 1] : v[e] * c[2 * e] + o[e] * c[2 * e + 1];
            }
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                const int j = j0 + e;
                v[e] = 0.0f;
                if (j < d.dim) {
                    v[e] = src[i0 + e];
                } else if (j < d.dim + d.rot) {
                    const int r = j - d.dim, p = r < half ? r : r - half;
                    const float2 f = cs[p];
                    const float* base = src + (i0 - j0) + d.dim;
                    const float a = base[p], b = base[p + half];
                    v[e] = r < half ? a * f.x - b * f.y : b * f.x + a * f.y;
                }
            }
        }
        store8(q + (long long)t * q_cols + i0, v);
        if (q_lat && j0 + 8 > d.dim && j0 < d.dim + d.rot) {
            T* dst = q_lat + ((long long)t * d.H + i0 / qh) * cr + d.rank - d.dim;  // (component j of the query -> rank + j - dim)
            if (vec && d.rank % 8 == 0) store8(dst + j0, v);
            else
#pragma unroll
                for (int e = 0; e < 8; ++e)
                    if (j0 + e >= d.dim && j0 + e < d.dim + d.rot) dst[j0 + e] = from_f32<T>(v[e]);
        }
        return;
    }
    // latent: RMS norm, then the cache entry
    const float* down = src + q_cols;
    float ss = 0.0f;
    for (int i = threadIdx.x; i < d.rank; i += 256) ss += down[i] * down[i];
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += red[w];
    const float rms = sqrtf(ss / (float)d.rank + eps);
    const int page = block_table[(long long)tok_row[t] * max_pages + pos / PAGE];
    T* dst = pool + ((long long)page * PAGE + pos % PAGE) * cr;
    for (int i = threadIdx.x; i < cr; i += 256) {
        float v = 0.0f;
        if (i < d.rank) {
            v = down[i] / rms * gain[i];
        } else if (i < d.rank + d.rot) {
            const int r = i - d.rank, p = r < half ? r : r - half;
            const float2 e = cs[p];
            const float a = down[d.rank + p], b = down[d.rank + p + half];
            v = r < half ? a * e.x - b * e.y : b * e.x + a * e.y;
        }
        dst[i] = from_f32<T>(v);
    }
}

// ---- per-head projections -----------------------------------------------------------------------------------------
// out[t][h][n] = sum_k in[t][h][k] * W[h][n][k], n < N, k < K; W rows of pitch kw (zero padded), W[h] of nw rows.
struct ProjectArgs {
    const void* in;
    long long in_ts, in_hs;
    const void* W;
    int N, K, nw, kw;
    void* out;
    long long out_ts, out_hs;
    int t0, T;
};

template <typename T>
__global__ void __launch_bounds__(256) latent_project_simt_kernel(ProjectArgs a) {
    chain_trigger();
    chain_wait();
    const int n = blockIdx.x * 32 + (threadIdx.x & 31), h = blockIdx.y;
    const int t = a.t0 + blockIdx.z * 8 + (threadIdx.x >> 5);
    if (t >= a.t0 + a.T || n >= a.N) return;
    const T* in = static_cast<const T*>(a.in) + t * a.in_ts + h * a.in_hs;
    float acc = 0.0f;
    const T* w = static_cast<const T*>(a.W) + ((long long)h * a.nw + n) * a.kw;
    for (int k = 0; k < a.K; ++k) acc = fmaf(to_f32(in[k]), to_f32(w[k]), acc);
    static_cast<T*>(a.out)[t * a.out_ts + h * a.out_hs + n] = from_f32<T>(acc);
}

// bf16 on the tensor cores: the weights are the 16-row operand, eight tokens the other, so that a decode step wastes no
// rows.  A lane's eight consecutive k of a 32-wide block feed two k16 products - both operands in the same order, so every
// fragment is one 16-byte load straight from global memory.  Four warps per CTA: 16 output rows each, or (KSPLIT) the same
// 16 rows and a quarter of k each, added in warp order; up to 32 tokens.
template <bool KSPLIT>
__global__ void __launch_bounds__(128) latent_project_mma_kernel(ProjectArgs a) {
    __shared__ float fold[KSPLIT ? 3 * 16 * 32 : 1];
    chain_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, h = blockIdx.y;
    const int n0 = KSPLIT ? blockIdx.x * 16 : blockIdx.x * 64 + warp * 16;
    const int g = lane >> 2, kq = (lane & 3) * 8;
    const int t_begin = a.t0 + blockIdx.z * 32, t_end = min(a.t0 + a.T, t_begin + 32);
    const int n_blk = a.kw / 32;
    const int b0 = KSPLIT ? n_blk * warp / 4 : 0, b1 = KSPLIT ? n_blk * (warp + 1) / 4 : n_blk;
    const bool on = n0 < a.N;
    const __nv_bfloat16* w0 = static_cast<const __nv_bfloat16*>(a.W) + ((long long)h * a.nw + (on ? n0 : 0) + g) * a.kw + kq;
    const __nv_bfloat16* w1 = w0 + 8 * a.kw;
    // the weights are constant: the first blocks are requested before the predecessor kernel has finished
    constexpr int PRE = 4;
    uint4 px[PRE], py[PRE];
#pragma unroll
    for (int i = 0; i < PRE; ++i)
        if (on && b0 + i < b1) {
            px[i] = __ldg(reinterpret_cast<const uint4*>(w0 + (b0 + i) * 32));
            py[i] = __ldg(reinterpret_cast<const uint4*>(w1 + (b0 + i) * 32));
        }
    chain_wait();
    float acc[4][4];
#pragma unroll
    for (int j = 0; j < 4; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
    if (on) {
        const __nv_bfloat16* in = static_cast<const __nv_bfloat16*>(a.in) + h * a.in_hs + kq;
        auto block = [&](int k, const uint4& x, const uint4& y) {
            const uint32_t a0[4] = {x.x, y.x, x.y, y.y}, a1[4] = {x.z, y.z, x.w, y.w};
            const bool k_in = k + kq < a.K;  // the operand's pitch covers K rounded up to 8; weights beyond K are zero
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (t_begin + j * 8 >= t_end) break;
                const int t = t_begin + j * 8 + g;
                uint4 b = make_uint4(0, 0, 0, 0);
                if (k_in && t < t_end) b = *reinterpret_cast<const uint4*>(in + t * a.in_ts + k);
                mma_16816(acc[j], a0, b.x, b.y);
                mma_16816(acc[j], a1, b.z, b.w);
            }
        };
#pragma unroll
        for (int i = 0; i < PRE; ++i)
            if (b0 + i < b1) block((b0 + i) * 32, px[i], py[i]);
#pragma unroll 4
        for (int i = b0 + PRE; i < b1; ++i)
            block(i * 32, __ldg(reinterpret_cast<const uint4*>(w0 + i * 32)), __ldg(reinterpret_cast<const uint4*>(w1 + i * 32)));
    }
    if constexpr (KSPLIT) {
        if (warp > 0)
#pragma unroll
            for (int j = 0; j < 4; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) fold[((warp - 1) * 16 + j * 4 + e) * 32 + lane] = acc[j][e];
        __syncthreads();
        if (warp == 0)
#pragma unroll
            for (int w = 0; w < 3; ++w)
#pragma unroll
                for (int j = 0; j < 4; ++j)
#pragma unroll
                    for (int e = 0; e < 4; ++e) acc[j][e] += fold[(w * 16 + j * 4 + e) * 32 + lane];
    }
    if (on && (!KSPLIT || warp == 0)) {
        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + h * a.out_hs;
#pragma unroll
        for (int j = 0; j < 4; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = t_begin + j * 8 + (lane & 3) * 2 + (e & 1), n = n0 + g + (e >> 1) * 8;
                if (t < t_end && n < a.N) out[t * a.out_ts + n] = __float2bfloat16_rn(acc[j][e]);
            }
    }
}

static jsm_status project(bool f32, const ProjectArgs& a, int H, cudaStream_t st) {
    if (a.T <= 0) return JSM_OK;
    if (f32)
        JSM_CUDA_CHECK(launch_chained(latent_project_simt_kernel<float>, dim3((a.N + 31) / 32, H, (a.T + 7) / 8), dim3(256), 0, st, a));
    else if (a.kw >= 256)
        JSM_CUDA_CHECK(launch_chained(latent_project_mma_kernel<true>, dim3((a.N + 15) / 16, H, (a.T + 31) / 32), dim3(128), 0, st, a));
    else
        JSM_CUDA_CHECK(launch_chained(latent_project_mma_kernel<false>, dim3((a.N + 63) / 64, H, (a.T + 31) / 32), dim3(128), 0, st, a));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

// ---- attention in the latent space --------------------------------------------------------------------------------
// Any sizes, f32 arithmetic throughout: one CTA per (token, head), online softmax over chunks of 128 keys.
template <typename T>
__global__ void __launch_bounds__(128) latent_attn_simt_kernel(const T* __restrict__ q_lat, LatentDims d, const T* __restrict__ pool,
                                                               const int32_t* __restrict__ block_table, int max_pages,
                                                               const int32_t* __restrict__ tok_row, const int32_t* __restrict__ tok_pos,
                                                               T* __restrict__ o_lat, int t_first) {
    extern __shared__ float sm[];
    const int cr = pad8(d.rank + d.rot), rp = pad8(d.rank), width = d.rank + d.rot;
    float* qs = sm;             // [cr]
    float* o = qs + cr;         // [rank]
    float* s = o + d.rank;      // [128]
    float* red = s + 128;       // [8]
    chain_trigger();
    chain_wait();
    const int t = t_first + blockIdx.x, h = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const T* qr = q_lat + ((long long)t * d.H + h) * cr;
    for (int i = threadIdx.x; i < cr; i += 128) qs[i] = to_f32(qr[i]);
    for (int i = threadIdx.x; i < d.rank; i += 128) o[i] = 0.0f;
    const int pos = tok_pos[t], k0 = max(0, pos - d.window + 1);
    const int32_t* bt = block_table + (long long)tok_row[t] * max_pages;
    float m = -INFINITY, l = 0.0f;
    for (int c0 = k0; c0 <= pos; c0 += 128) {
        const int n = min(128, pos + 1 - c0);
        __syncthreads();
        for (int j = warp; j < n; j += 4) {
            const int kp = c0 + j;
            const T* e = pool + ((long long)bt[kp / PAGE] * PAGE + kp % PAGE) * cr;
            float acc = 0.0f;
            for (int i = lane; i < width; i += 32) acc = fmaf(qs[i], to_f32(e[i]), acc);
            acc = warp_sum(acc);
            if (lane == 0) s[j] = acc * d.scale;
        }
        __syncthreads();
        float v = threadIdx.x < n ? s[threadIdx.x] : -INFINITY;
        float mx = warp_max(v);
        if (lane == 0) red[warp] = mx;
        __syncthreads();
        mx = fmaxf(fmaxf(red[0], red[1]), fmaxf(red[2], red[3]));
        const float m_new = fmaxf(m, mx), alpha = expf(m - m_new);
        const float p = threadIdx.x < n ? expf(v - m_new) : 0.0f;
        s[threadIdx.x] = p;
        const float ps = warp_sum(p);
        if (lane == 0) red[4 + warp] = ps;
        __syncthreads();
        l = l * alpha + ((red[4] + red[5]) + (red[6] + red[7]));
        m = m_new;
        for (int i = threadIdx.x; i < d.rank; i += 128) {
            float acc = o[i] * alpha;
            for (int j = 0; j < n; ++j) {
                const int kp = c0 + j;
                acc = fmaf(s[j], to_f32(pool[((long long)bt[kp / PAGE] * PAGE + kp % PAGE) * cr + i]), acc);
            }
            o[i] = acc;
        }
    }
    T* out = o_lat + ((long long)t * d.H + h) * rp;
    for (int i = threadIdx.x; i < rp; i += 128) out[i] = from_f32<T>(i < d.rank ? o[i] / l : 0.0f);
}

// bf16 on the tensor cores.  A CTA owns 32 (token, head) rows of one segment and a run of cache pages; a page of 64 entries
// is one stage of a two-stage ring filled by bulk copies (a row each), read once for the scores (all
// rank + rot components) and once for the weighted sum (the first rank components).  Eight warps: scores as 2 tiles of 16
// rows x 2 halves of the components x 2 groups of 32 keys - a warp keeps its part of the queries in registers - then the sum
// as column blocks of NT x 8 latent components per warp, all 32 rows.  Scores, maxima and sums are fp32; the weights enter the
// sum as bf16.  Waits for copies are bounded (tc_utils.cuh).
constexpr int LA_ROWS = LATENT_TILE_ROWS;
constexpr int LA_SP = 68;  // pitch of the score tile (floats)
constexpr int LA_PP = 72;  // pitch of the weight tile (bf16)
constexpr int LA_ML = 4;   // behind a partial row: its maximum, its sum, two unused
constexpr int LA_MAX_SPLITS = 128;
constexpr int LA_ERR_FULL = 51;

static int la_pitch(const LatentDims& d) { return pad_to(d.rank + d.rot, 16) + 8; }  // odd multiple of 16 bytes: no bank conflicts
static size_t la_smem(const LatentDims& d) {
    return (size_t)2 * PAGE * la_pitch(d) * 2 + LA_ROWS * LA_PP * 2 + 2 * LA_ROWS * LA_SP * 4 + 3 * LA_ROWS * 4;
}

template <int NT>  // KS: 16-wide steps of half the components, at most
__global__ void __launch_bounds__(256, 1) latent_attn_mma_kernel(const __nv_bfloat16* __restrict__ q_lat, LatentDims d,
                                                              const __nv_bfloat16* __restrict__ pool, const int32_t* __restrict__ block_table,
                                                              int max_pages, const int32_t* __restrict__ seg_start,
                                                              const int32_t* __restrict__ seg_len, const int32_t* __restrict__ seg_pos0,
                                                              const int32_t* __restrict__ seg_row, const int32_t* __restrict__ tile_seg,
                                                              const int32_t* __restrict__ tile_r0, __nv_bfloat16* __restrict__ o_lat,
                                                              float* __restrict__ part, int splits, int pitch, int* err) {
    constexpr int KS = 2 * NT + 4;
    extern __shared__ __align__(16) uint8_t la_dyn[];
    __nv_bfloat16* kv = reinterpret_cast<__nv_bfloat16*>(la_dyn);       // 2 x [64][pitch]
    __nv_bfloat16* ps = kv + 2 * PAGE * pitch;                          // [32][72]
    float* ss = reinterpret_cast<float*>(ps + LA_ROWS * LA_PP);         // 2 x [32][68]: halves of the components
    float* row_m = ss + 2 * LA_ROWS * LA_SP;
    float* row_l = row_m + LA_ROWS;
    float* row_a = row_l + LA_ROWS;
    __shared__ __align__(8) uint64_t full[2];
    __shared__ int abort_flag;
    chain_trigger();
    const int cr = pad8(d.rank + d.rot), rp = pad8(d.rank), cr16 = pitch - 8;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (threadIdx.x == 0) {
        abort_flag = 0;
        tc::mbar_init(&full[0], 1);
        tc::mbar_init(&full[1], 1);
        tc::mbar_fence_init();
    }
    // columns between the entry's pitch and the next multiple of 16 take part in the products: zero once
    if (cr < cr16)
        for (int i = threadIdx.x; i < 2 * PAGE * (cr16 - cr); i += 256) kv[(i / (cr16 - cr)) * pitch + cr + i % (cr16 - cr)] = __float2bfloat16_rn(0.0f);
    if (threadIdx.x < LA_ROWS) { row_m[threadIdx.x] = -INFINITY; row_l[threadIdx.x] = 0.0f; }
    __syncthreads();
    chain_wait();
    const int tile = blockIdx.x, sp = blockIdx.y;
    const int seg = tile_seg[tile], r0 = tile_r0[tile];
    const int start = seg_start[seg], len = seg_len[seg], pos0 = seg_pos0[seg];
    const int n_rows = min(LA_ROWS, len * d.H - r0);
    const int p_first = pos0 + r0 / d.H, p_last = pos0 + (r0 + n_rows - 1) / d.H;
    const int key_lo = max(0, p_first - d.window + 1), key_hi = p_last + 1;
    const int pg_lo = key_lo / PAGE, n_pg = (key_hi - 1) / PAGE - pg_lo + 1;
    const int live = min(splits, n_pg);  // the grid is made for the longest context: the splits behind the pages of this one rest
    if (sp >= live) return;
    const int pb = pg_lo + n_pg * sp / live, pe = pg_lo + n_pg * (sp + 1) / live;
    const int32_t* bt = block_table + (long long)seg_row[seg] * max_pages;
    const int vec = cr / 8;  // 16-byte vectors per entry
    // A row per copy, issued by the first eight lanes of every warp (a thread's copies go out one after the other, and one
    // warp would hold up the others).  A copy that lands before the expected bytes are announced cannot complete the phase:
    // the announcement is also its only arrival.
    auto load_page = [&](int pg, int stage) {
        const int lo = max(key_lo - pg * PAGE, 0), hi = min(key_hi - pg * PAGE, PAGE);
        if (threadIdx.x == 0) tc::mbar_expect_tx(&full[stage], (uint32_t)(hi - lo) * cr * 2);
        const int r = warp * 8 + lane;
        if (lane < 8 && r >= lo && r < hi)
            asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];" ::"r"(
                             smem_u32(kv + (stage * PAGE + r) * pitch)),
                         "l"(reinterpret_cast<uint64_t>(pool + ((long long)bt[pg] * PAGE + r) * cr)), "r"(cr * 2), "r"(smem_u32(&full[stage]))
                         : "memory");
    };
    load_page(pb, 0);
    // the queries pass through the second stage into registers
    for (int i = threadIdx.x; i < LA_ROWS * vec; i += 256) {
        const int r = i / vec, c = i - r * vec, g = r0 + r;
        const int t = start + g / d.H, h = g % d.H;
        cp_async16(smem_u32(kv + (PAGE + r) * pitch + c * 8), q_lat + ((long long)(r < n_rows ? t : start) * d.H + (r < n_rows ? h : 0)) * cr + c * 8, r < n_rows);
    }
    cp_async_commit();
    cp_async_wait<0>();
    __syncthreads();
    const int mt = warp & 1, kh = (warp >> 1) & 1, kg = warp >> 2;  // this warp's rows, half of the components, keys
    const int lm = lane >> 3, lr = lane & 7;
    const int n_ks = cr16 / 16, ks0 = kh ? (n_ks + 1) / 2 : 0, n_mine = kh ? n_ks / 2 : (n_ks + 1) / 2;
    uint32_t qf[KS][4];
    {
        const uint32_t q_addr = smem_u32(kv + (PAGE + mt * 16 + (lm & 1) * 8 + lr) * pitch + (lm >> 1) * 8);
#pragma unroll
        for (int k = 0; k < KS; ++k)
            if (k < n_mine) ldsm_x4(q_addr + (ks0 + k) * 32, qf[k]);
    }
    tc::fence_proxy_async_smem();  // the copy engine writes this stage next
    __syncthreads();
    float o[2][NT][4];
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int j = 0; j < NT; ++j) o[a][j][0] = o[a][j][1] = o[a][j][2] = o[a][j][3] = 0.0f;
    bool ok = true;
    for (int pg = pb; pg < pe; ++pg) {
        const int i = pg - pb, stage = i & 1;
        if (pg + 1 < pe) load_page(pg + 1, stage ^ 1);
        __nv_bfloat16* kvs = kv + stage * PAGE * pitch;
        {   // entries outside the tile's key range are not fetched: their rows are zero (a weight of 0 must meet a number)
            const int lo = max(key_lo - pg * PAGE, 0), hi = min(key_hi - pg * PAGE, PAGE);
            if (lo > 0 || hi < PAGE) {
                const int n_out = lo + PAGE - hi;
                for (int q = threadIdx.x; q < n_out * vec; q += 256) {
                    const int r = q / vec, c = q - r * vec;
                    *reinterpret_cast<uint4*>(kvs + (r < lo ? r : hi + r - lo) * pitch + c * 8) = make_uint4(0, 0, 0, 0);
                }
                tc::fence_proxy_async_smem();
            }
        }
        ok = tc::mbar_wait(&full[stage], (i >> 1) & 1, &abort_flag, err, LA_ERR_FULL);
        if (!__syncthreads_and(ok)) { ok = false; break; }
        {   // scores
            float s[4][4];
#pragma unroll
            for (int j = 0; j < 4; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.0f;
            const uint32_t k_addr = smem_u32(kvs + (kg * 32 + (lm >> 1) * 8 + lr) * pitch + (lm & 1) * 8) + ks0 * 32;
#pragma unroll
            for (int k = 0; k < KS; ++k)
                if (k < n_mine) {
                    uint32_t b0[4], b1[4];
                    ldsm_x4(k_addr + k * 32, b0);
                    ldsm_x4(k_addr + 16 * pitch * 2 + k * 32, b1);
                    mma_16816(s[0], qf[k], b0[0], b0[1]);
                    mma_16816(s[1], qf[k], b0[2], b0[3]);
                    mma_16816(s[2], qf[k], b1[0], b1[1]);
                    mma_16816(s[3], qf[k], b1[2], b1[3]);
                }
            float* dst = ss + (kh * LA_ROWS + mt * 16 + (lane >> 2)) * LA_SP + kg * 32 + (lane & 3) * 2;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                *reinterpret_cast<float2*>(dst + j * 8) = make_float2(s[j][0], s[j][1]);
                *reinterpret_cast<float2*>(dst + 8 * LA_SP + j * 8) = make_float2(s[j][2], s[j][3]);
            }
        }
        __syncthreads();
        {   // softmax: a warp takes four rows side by side, two keys per lane
            constexpr int R = LA_ROWS / 8;
            float a[R], b[R], mx[R], sum[R], m_old[R], ref[R];
#pragma unroll
            for (int q = 0; q < R; ++q) {
                const int r = warp * R + q, p = pos0 + (r0 + r) / d.H, k0 = pg * PAGE + lane, k1 = k0 + 32;
                const bool on = r < n_rows;
                const float* sr = ss + r * LA_SP + lane;
                a[q] = (on && k0 <= p && p - k0 < d.window) ? (sr[0] + sr[LA_ROWS * LA_SP]) * d.scale : -INFINITY;
                b[q] = (on && k1 <= p && p - k1 < d.window) ? (sr[32] + sr[LA_ROWS * LA_SP + 32]) * d.scale : -INFINITY;
                mx[q] = fmaxf(a[q], b[q]);
                m_old[q] = row_m[r];
            }
#pragma unroll
            for (int x = 16; x > 0; x >>= 1)
#pragma unroll
                for (int q = 0; q < R; ++q) mx[q] = fmaxf(mx[q], __shfl_xor_sync(0xffffffffu, mx[q], x));
#pragma unroll
            for (int q = 0; q < R; ++q) {
                mx[q] = fmaxf(mx[q], m_old[q]);
                ref[q] = mx[q] == -INFINITY ? 0.0f : mx[q];
                a[q] = __expf(a[q] - ref[q]);
                b[q] = __expf(b[q] - ref[q]);
                sum[q] = a[q] + b[q];
                ps[(warp * R + q) * LA_PP + lane] = __float2bfloat16_rn(a[q]);
                ps[(warp * R + q) * LA_PP + lane + 32] = __float2bfloat16_rn(b[q]);
            }
#pragma unroll
            for (int x = 16; x > 0; x >>= 1)
#pragma unroll
                for (int q = 0; q < R; ++q) sum[q] += __shfl_xor_sync(0xffffffffu, sum[q], x);
            if (lane == 0)
#pragma unroll
                for (int q = 0; q < R; ++q) {
                    const int r = warp * R + q;
                    const float al = __expf(m_old[q] - ref[q]);
                    row_a[r] = al;
                    row_l[r] = row_l[r] * al + sum[q];
                    row_m[r] = mx[q];
                }
        }
        __syncthreads();
        // weighted sum of the latents
#pragma unroll
        for (int a = 0; a < 2; ++a) {
            const float al0 = row_a[a * 16 + (lane >> 2)], al1 = row_a[a * 16 + (lane >> 2) + 8];
#pragma unroll
            for (int j = 0; j < NT; ++j) { o[a][j][0] *= al0; o[a][j][1] *= al0; o[a][j][2] *= al1; o[a][j][3] *= al1; }
        }
        const int col0 = warp * NT * 8;
        if (col0 < d.rank) {
#pragma unroll
            for (int k = 0; k < PAGE; k += 16) {
                uint32_t p0[4], p1[4];
                ldsm_x4(smem_u32(ps + ((lm & 1) * 8 + lr) * LA_PP + k + (lm >> 1) * 8), p0);
                ldsm_x4(smem_u32(ps + (16 + (lm & 1) * 8 + lr) * LA_PP + k + (lm >> 1) * 8), p1);
#pragma unroll
                for (int j = 0; j < NT; j += 2) {
                    const int c = col0 + j * 8;
                    if (c < d.rank) {
                        uint32_t v[4];
                        ldsm_x4_trans(smem_u32(kvs + (k + (lm & 1) * 8 + lr) * pitch + c + (lm >> 1) * 8), v);
                        mma_16816(o[0][j], p0, v[0], v[1]);
                        mma_16816(o[1][j], p1, v[0], v[1]);
                        mma_16816(o[0][j + 1], p0, v[2], v[3]);
                        mma_16816(o[1][j + 1], p1, v[2], v[3]);
                    }
                }
            }
        }
        __syncthreads();  // the stage and the score / weight tiles are free
    }
    if (!ok) {  // a copy did not arrive: let the ones in flight land (bounded) and leave the result undefined; the host learns of it
        if (threadIdx.x == 0) {
            const long long t0 = clock64();
            while (clock64() - t0 < tc::WAIT_LIMIT_CYCLES / 4) {}
        }
        __syncthreads();
        return;
    }
    // rows whose keys all lie in other splits have l = 0, m = -inf: they weigh nothing in the merge
#pragma unroll
    for (int a = 0; a < 2; ++a)
#pragma unroll
        for (int e = 0; e < 4; e += 2) {
            const int r = a * 16 + (lane >> 2) + (e >> 1) * 8;
            if (r >= n_rows) continue;
            const int g = r0 + r;
            const float inv = splits == 1 ? 1.0f / row_l[r] : 1.0f;
#pragma unroll
            for (int j = 0; j < NT; ++j) {
                const int c = (warp * NT + j) * 8 + (lane & 3) * 2;
                if (splits == 1) {
                    if (c < rp) {  // (rp is a multiple of 8: a pair never straddles it)
                        __nv_bfloat16* out = o_lat + ((long long)(start + g / d.H) * d.H + g % d.H) * rp;
                        *reinterpret_cast<uint32_t*>(out + c) =
                            pack_bf16x2(c < d.rank ? o[a][j][e] * inv : 0.0f, c + 1 < d.rank ? o[a][j][e + 1] * inv : 0.0f);
                    }
                } else {
                    float* out = part + (((long long)tile * splits + sp) * LA_ROWS + r) * (rp + LA_ML);
                    if (c < rp) *reinterpret_cast<float2*>(out + c) = make_float2(o[a][j][e], o[a][j][e + 1]);
                    if (warp == 0 && j == 0 && (lane & 3) == 0) { out[rp] = row_m[r]; out[rp + 1] = row_l[r]; }
                }
            }
        }
}

// merges the partials of the splits in split order; one CTA per (tile, row), four columns per thread
__global__ void __launch_bounds__(128) latent_combine_kernel(const float* __restrict__ part, LatentDims d, const int32_t* __restrict__ seg_start,
                                                             const int32_t* __restrict__ seg_len, const int32_t* __restrict__ tile_seg,
                                                             const int32_t* __restrict__ seg_pos0, const int32_t* __restrict__ tile_r0, int max_splits,
                                                             __nv_bfloat16* __restrict__ o_lat) {
    chain_trigger();
    chain_wait();
    const int tile = blockIdx.x, r = blockIdx.y, rp = pad8(d.rank), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int seg = tile_seg[tile], g = tile_r0[tile] + r;
    const int r0 = tile_r0[tile], n_all = seg_len[seg] * d.H;
    if (g >= n_all) return;
    // the splits that had pages (as in the attention kernel)
    const int p_first = seg_pos0[seg] + r0 / d.H, p_last = seg_pos0[seg] + (min(r0 + LA_ROWS, n_all) - 1) / d.H;
    const int splits = min(max_splits, p_last / PAGE - max(0, p_first - d.window + 1) / PAGE + 1);
    const long long stride = (long long)LA_ROWS * (rp + LA_ML);
    const float* p = part + ((long long)tile * max_splits * LA_ROWS + r) * (rp + LA_ML);
    // every warp works out the weights for itself: lane s % 32 holds those of split s
    float ms[LA_MAX_SPLITS / 32], w[LA_MAX_SPLITS / 32], m = -INFINITY, l = 0.0f;
#pragma unroll
    for (int i = 0; i < LA_MAX_SPLITS / 32; ++i) {
        ms[i] = -INFINITY; w[i] = 0.0f;
        const int s = i * 32 + lane;
        if (s < splits) {
            const float2 v = *reinterpret_cast<const float2*>(p + s * stride + rp);
            ms[i] = v.x; w[i] = v.y;
            m = fmaxf(m, v.x);
        }
    }
    m = warp_max(m);
#pragma unroll
    for (int i = 0; i < LA_MAX_SPLITS / 32; ++i) {
        const float e = __expf(ms[i] - m);
        l += e * w[i];
        w[i] = e;
    }
    const float inv = 1.0f / warp_sum(l);
    __nv_bfloat16* out = o_lat + ((long long)(seg_start[seg] + g / d.H) * d.H + g % d.H) * rp;
    for (int c0 = warp * 128; c0 < rp; c0 += 512) {  // (warp-uniform: the shuffles need every lane)
        const int c = c0 + lane * 4, cc = min(c, rp - 4);
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < LA_MAX_SPLITS / 32; ++i) {
            if (i * 32 >= splits) break;
            const int n = min(32, splits - i * 32);
#pragma unroll 8
            for (int s = 0; s < n; ++s) {
                const float4 v = __ldcs(reinterpret_cast<const float4*>(p + (i * 32 + s) * stride + cc));
                const float f = __shfl_sync(0xffffffffu, w[i], s);  // a split without a visible key holds zeros and weighs nothing
                acc.x = fmaf(f, v.x, acc.x); acc.y = fmaf(f, v.y, acc.y); acc.z = fmaf(f, v.z, acc.z); acc.w = fmaf(f, v.w, acc.w);
            }
        }
        if (c < rp) {
            uint2 u;
            u.x = pack_bf16x2(c < d.rank ? acc.x * inv : 0.0f, c + 1 < d.rank ? acc.y * inv : 0.0f);
            u.y = pack_bf16x2(c + 2 < d.rank ? acc.z * inv : 0.0f, c + 3 < d.rank ? acc.w * inv : 0.0f);
            *reinterpret_cast<uint2*>(out + c) = u;
        }
    }
}

__global__ void __launch_bounds__(256) latent_gather_kernel(const __nv_bfloat16* __restrict__ pool, const int32_t* __restrict__ bt, int p0, int n,
                                                            int vec, uint4* __restrict__ out) {
    chain_trigger();
    chain_wait();
    const long long total = (long long)n * vec;
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < total; i += (long long)gridDim.x * 256) {
        const int r = (int)(i / vec), c = (int)(i - (long long)r * vec), p = p0 + r;
        out[i] = reinterpret_cast<const uint4*>(pool)[((long long)bt[p / PAGE] * PAGE + p % PAGE) * vec + c];
    }
}

// ---- launches -----------------------------------------------------------------------------------------------------
jsm_status latent_prep_launch(bool f32, const float* qd, const LatentDims& d, const LatentWeights& w, float eps, const LatentCache& cache,
                              const StepTokens& tk, void* q, void* q_lat, cudaStream_t st) {
    const dim3 grid(tk.T, (d.q_cols() / 8 + 255) / 256 + 1);
    const int vec = d.dim % 8 == 0 && d.rot % 16 == 0 ? 1 : 0;
    if (f32)
        JSM_CUDA_CHECK(launch_chained(latent_prep_kernel<float>, grid, dim3(256), 0, st, qd, d, w.down_norm, eps, (float*)cache.pool,
                                      cache.block_table, cache.max_pages, cache.rope, tk.tok_row, tk.tok_pos, (float*)q, (float*)q_lat, vec));
    else
        JSM_CUDA_CHECK(launch_chained(latent_prep_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, qd, d, w.down_norm, eps,
                                      (__nv_bfloat16*)cache.pool, cache.block_table, cache.max_pages, cache.rope, tk.tok_row, tk.tok_pos,
                                      (__nv_bfloat16*)q, (__nv_bfloat16*)q_lat, vec));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

static int la_nt(const LatentDims& d) { return d.rank <= 128 ? 2 : d.rank <= 256 ? 4 : d.rank <= 384 ? 6 : 8; }
bool latent_mma_usable(const LatentDims& d) {
    // a warp's half of the queries: at most 2 NT + 4 steps of 16 components
    return d.rank <= 512 && (pad_to(d.rank + d.rot, 16) / 16 + 1) / 2 <= 2 * la_nt(d) + 4 && la_smem(d) <= 226 * 1024;
}

int latent_splits(int n_tiles, int max_keys) {
    if (n_tiles <= 0) return 1;
    const int pages = max_keys / PAGE + 2;
    return std::max(1, std::min({sm_count() / n_tiles, pages / 2, LA_MAX_SPLITS}));
}
size_t latent_part_floats(const LatentDims& d) { return (size_t)sm_count() * LA_ROWS * (pad8(d.rank) + LA_ML); }

template <int NT>
static jsm_status launch_mma(const LatentDims& d, const LatentCache& cache, const StepTokens& tk, const LatentTiles& tl, const LatentScratch& sc,
                             int splits, cudaStream_t st) {
    static bool attr_done = false;
    if (!attr_done) {
        JSM_CUDA_CHECK(cudaFuncSetAttribute(latent_attn_mma_kernel<NT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 226 * 1024));
        attr_done = true;
    }
    JSM_CUDA_CHECK(launch_chained(latent_attn_mma_kernel<NT>, dim3(tl.n_tiles, splits), dim3(256), la_smem(d), st, (const __nv_bfloat16*)sc.q_lat, d,
                                  (const __nv_bfloat16*)cache.pool, cache.block_table, cache.max_pages, tk.seg_start, tk.seg_len, tk.seg_pos0,
                                  tk.seg_row, tl.tile_seg, tl.tile_r0, (__nv_bfloat16*)sc.o_lat, sc.part, splits, la_pitch(d), tc_error_word()));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

jsm_status latent_attn_launch(bool f32, const LatentDims& d, const LatentWeights& w, const LatentCache& cache, const StepTokens& tk,
                              const LatentTiles& tl, const void* q, const LatentScratch& sc, void* out, cudaStream_t st) {
    if (tl.n_tiles <= 0 || tl.t_count <= 0) return JSM_OK;
    const int cr = d.cr(), rp = pad8(d.rank);
    ProjectArgs a;
    a.in = q; a.in_ts = d.q_cols(); a.in_hs = d.qh();
    a.W = w.uk; a.N = d.rank; a.K = d.dim; a.nw = pad_to(d.rank, 16); a.kw = pad_to(d.dim, 32);
    a.out = sc.q_lat; a.out_ts = (long long)d.H * cr; a.out_hs = cr;
    a.t0 = tl.t_first; a.T = tl.t_count;
    jsm_status s = project(f32, a, d.H, st);
    if (s != JSM_OK) return s;
    if (f32 || !latent_mma_usable(d)) {
        const size_t smem = sizeof(float) * (cr + d.rank + 128 + 8);
        if (smem > 48 * 1024) JSM_FAIL(JSM_UNSUPPORTED, "latent attention: latent of %d + %d components", d.rank, d.rot);
        if (f32)
            JSM_CUDA_CHECK(launch_chained(latent_attn_simt_kernel<float>, dim3(tl.t_count, d.H), dim3(128), smem, st, (const float*)sc.q_lat, d,
                                          (const float*)cache.pool, cache.block_table, cache.max_pages, tk.tok_row, tk.tok_pos, (float*)sc.o_lat,
                                          tl.t_first));
        else
            JSM_CUDA_CHECK(launch_chained(latent_attn_simt_kernel<__nv_bfloat16>, dim3(tl.t_count, d.H), dim3(128), smem, st,
                                          (const __nv_bfloat16*)sc.q_lat, d, (const __nv_bfloat16*)cache.pool, cache.block_table, cache.max_pages,
                                          tk.tok_row, tk.tok_pos, (__nv_bfloat16*)sc.o_lat, tl.t_first));
        JSM_LAUNCH_CHECK();
    } else {
        const int splits = latent_splits(tl.n_tiles, tl.max_keys);
        if (splits > 1 && (size_t)tl.n_tiles * splits * LA_ROWS * (rp + LA_ML) > sc.part_floats)
            JSM_FAIL(JSM_INVALID_ARG, "latent attention: workspace of %zu floats for %d tiles in %d splits", sc.part_floats, tl.n_tiles, splits);
        switch (la_nt(d)) {
            case 2: s = launch_mma<2>(d, cache, tk, tl, sc, splits, st); break;
            case 4: s = launch_mma<4>(d, cache, tk, tl, sc, splits, st); break;
            case 6: s = launch_mma<6>(d, cache, tk, tl, sc, splits, st); break;
            default: s = launch_mma<8>(d, cache, tk, tl, sc, splits, st); break;
        }
        if (s != JSM_OK) return s;
        if (splits > 1) {
            JSM_CUDA_CHECK(launch_chained(latent_combine_kernel, dim3(tl.n_tiles, LA_ROWS), dim3(128), 0, st, (const float*)sc.part, d, tk.seg_start,
                                          tk.seg_len, tl.tile_seg, tk.seg_pos0, tl.tile_r0, splits, (__nv_bfloat16*)sc.o_lat));
            JSM_LAUNCH_CHECK();
        }
    }
    // values: out[t][h * vdim + j] = Wuv[h][j] . o_lat[t][h]
    a.in = sc.o_lat; a.in_ts = (long long)d.H * rp; a.in_hs = rp;
    a.W = w.uv; a.N = d.vdim; a.K = d.rank; a.nw = pad_to(d.vdim, 16); a.kw = pad_to(d.rank, 32);
    a.out = out; a.out_ts = d.out_cols(); a.out_hs = d.vdim;
    return project(f32, a, d.H, st);
}

jsm_status latent_gather_launch(const LatentDims& d, const LatentCache& cache, int row, int p0, int n, void* out, cudaStream_t st) {
    if (n <= 0) return JSM_OK;
    const int vec = d.cr() / 8;
    const long long total = (long long)n * vec;
    const int blocks = (int)std::min<long long>((total + 255) / 256, (long long)sm_count() * 8);
    JSM_CUDA_CHECK(launch_chained(latent_gather_kernel, dim3(blocks), dim3(256), 0, st, (const __nv_bfloat16*)cache.pool,
                                  cache.block_table + (long long)row * cache.max_pages, p0, n, vec, (uint4*)out));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

}  // namespace jsm
