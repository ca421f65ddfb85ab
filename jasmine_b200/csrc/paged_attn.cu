// Grouped-query attention over a paged cache, with the parts a design can switch on: biases of the projections, RMS norm of
// queries and keys per head, rotation of adjacent pairs on the first components, a mask (full, sliding window, chunks of the
// sequence), a learned sink in the softmax denominator, a gate per head on the output.  A layer without keys and values of
// its own reads another layer's cache.
//
// Cache: a page holds 64 positions; the keys and values of one kv head in a page are one contiguous block of 64-column slabs
// (keys first, then values), [slab][64 positions][64 columns] with columns behind the head's zero.  The 16-byte pieces of a
// slab's rows lie in the 128-byte swizzle of the tensor core's shared-memory tiles, so that a block is fetched by one plain
// bulk copy and used where it lands: here for decode steps and short portions, by the flash kernel (flash_attn.cu) for long
// ones.  A page's first token also clears the values behind the last one, so that a weight of zero always meets a number.
//
// Kernels: attn_prep (bias, norm, rotation, append, gates), attn_paged_mma (decode steps and short portions of bf16 models:
// keys as the 16-row operand, queries of the group as columns, split over the pages, the last CTA merges), attn_paged_simt
// (f32 models and heads wider than 256).
#include "decoder_ops.cuh"
#include "mma_utils.cuh"
#include "tc_utils.cuh"
#include <math.h>
#include <algorithm>

namespace jsm {

using tc::smem_u32;

constexpr int PAGE = JSM_PAGE_SIZE;
constexpr int SLAB = PAGE * 64;  // elements of a slab

// element (key, column) of a slab
template <typename T>
__device__ __forceinline__ int slab_index(int key, int col) { return key * 64 + ((((col >> 3) & 7) ^ (key & 7)) << 3) + (col & 7); }
// value: 0 keys, 1 values
template <typename T>
__device__ __forceinline__ T* cache_at(T* pool, const AttnDims& d, int page, int g, int value, int key, int col) {
    return pool + ((long long)(page * d.G + g) * (d.ks() + d.vs()) + (value ? d.ks() : 0) + (col >> 6)) * SLAB + slab_index<T>(key, col);
}

// ---- bias, norm, rotation, append ---------------------------------------------------------------------------------
// A warp takes one unit of TOK consecutive tokens: the query heads, then the key heads, the value heads (own_kv), and one unit
// for the gates.  wide row of a token: [q | gates | k | v].  NP: pairs of components per lane (0: any number, read twice).
template <typename T, int NP, int TOK>
__global__ void __launch_bounds__(256) attn_prep_kernel(const float* __restrict__ wide, AttnDims d, AttnWeights w, float eps, T* __restrict__ pool,
                                                        const int32_t* __restrict__ block_table, int max_pages, const float2* __restrict__ rope,
                                                        const int32_t* __restrict__ tok_row, const int32_t* __restrict__ tok_pos, int own_kv, int n_tok,
                                                        T* __restrict__ q, float* __restrict__ gate) {
    static_assert(NP > 0 || TOK == 1, "heads of any width take one token");
    const int t0 = blockIdx.x * TOK, unit = blockIdx.y * 8 + (threadIdx.x >> 5), lane = threadIdx.x & 31;
    const int kv_units = own_kv ? 2 * d.G : 0;
    const int off = d.q_cols() + pad8(d.H), pitch = d.wide_cols(own_kv != 0);
    chain_trigger();
    chain_wait();
    if (unit >= d.H + kv_units + d.gated) return;
    if (unit == d.H + kv_units) {
        for (int t = t0; t < min(n_tok, t0 + TOK); ++t)
            for (int h = lane; h < d.H; h += 32) gate[(long long)t * d.H + h] = 1.0f / (1.0f + expf(-wide[(long long)t * pitch + d.q_cols() + h]));
        return;
    }
    auto put = [](T* dst, const float2& v) {
        if constexpr (sizeof(T) == 2) *reinterpret_cast<uint32_t*>(dst) = pack_bf16x2(v.x, v.y);
        else *reinterpret_cast<float2*>(dst) = v;
    };
    const bool value = unit >= d.H + d.G, key = unit >= d.H && !value;
    const int hd = value ? unit - d.H - d.G : key ? unit - d.H : unit;
    const int n = value ? d.vdim : d.dim;
    const int col0 = value ? off + d.G * d.qh() + hd * pad8(d.vdim) : (key ? off : 0) + hd * d.qh();  // of the unit in a row
    const int end = value ? d.vs() * 32 : key ? d.ks() * 32 : d.qh() / 2;                              // pairs to write
    const float* bias = value ? w.v_bias : key ? w.k_bias : w.q_bias;
    if (bias) bias += hd * (value ? pad8(d.vdim) : d.qh());
    const float* gain = value ? nullptr : key ? w.k_norm : w.q_norm;
    // (the pitch of a head is a multiple of 8: a pair lies inside it, and bias and gain are zero behind the head)
    auto vec = [&](const float* p, int pr, float none) { return p && 2 * pr < n ? *reinterpret_cast<const float2*>(p + 2 * pr) : make_float2(none, none); };
    auto pair = [&](int t, int pr, const float2& b) {
        float2 v = vec(wide + (long long)t * pitch + col0, pr, 0.0f);
        v.x += b.x; v.y += b.y;
        if (2 * pr + 1 >= n) v.y = 0.0f;
        return v;
    };
    // where pair pr of a token goes
    auto entry = [&](int t, int pos) {  // keys and values: first element of the token's row in the first slab
        return cache_at(pool, d, block_table[(long long)tok_row[t] * max_pages + pos / PAGE], hd, value ? 1 : 0, pos % PAGE, 0) - slab_index<T>(pos % PAGE, 0) + pos % PAGE * 64;
    };
    auto store = [&](T* row, int pos, int pr, const float2& v) {
        put(key || value ? row + (pr >> 5) * SLAB + ((((pr >> 2) & 7) ^ (pos & 7)) << 3) + (pr & 3) * 2 : row + 2 * pr, v);
    };
    auto turn = [&](int pos, int pr, float2 v, float inv, const float2& g) {
        v.x *= inv * g.x; v.y *= inv * g.y;
        if (2 * pr < d.rot) {
            const float2 e = rope[pos * (d.rot / 2) + pr];
            v = make_float2(v.x * e.x - v.y * e.y, v.y * e.x + v.x * e.y);
        }
        return v;
    };
    auto length = [&](float ss) { return gain ? 1.0f / sqrtf(warp_sum(ss) / (float)n + eps) : 1.0f; };
    if (value) {
        for (int i = 0; i < TOK; ++i) {
            const int t = t0 + i;
            if (t >= n_tok) break;
            const int pos = tok_pos[t], in = pos % PAGE, r = tok_row[t];
            T* row = entry(t, pos);
            for (int pr = lane; pr < end; pr += 32) store(row, pos, pr, pair(t, pr, vec(bias, pr, 0.0f)));
            // last token of its portion, in a page that this portion opened: clear the rest of the page's values
            const bool last = t + 1 == n_tok || tok_row[t + 1] != r;
            if (last && t >= in && tok_row[t - in] == r && tok_pos[t - in] == pos - in)
                for (int s = 0; s < d.vs(); ++s)
                    for (int k = 64 + lane * 2; k < SLAB - in * 64; k += 64) put(row + s * SLAB + k, make_float2(0.0f, 0.0f));
        }
    } else if constexpr (NP > 0) {
        float2 v[TOK][NP], g[NP];
        {
            float2 b[NP];
#pragma unroll
            for (int k = 0; k < NP; ++k) { b[k] = vec(bias, k * 32 + lane, 0.0f); g[k] = vec(gain, k * 32 + lane, 1.0f); }
#pragma unroll
            for (int i = 0; i < TOK; ++i)
#pragma unroll
                for (int k = 0; k < NP; ++k) v[i][k] = t0 + i < n_tok ? pair(t0 + i, k * 32 + lane, b[k]) : make_float2(0.0f, 0.0f);
        }
#pragma unroll
        for (int i = 0; i < TOK; ++i) {
            const int t = t0 + i;
            if (t >= n_tok) break;
            float ss = 0.0f;
#pragma unroll
            for (int k = 0; k < NP; ++k) ss = fmaf(v[i][k].x, v[i][k].x, fmaf(v[i][k].y, v[i][k].y, ss));
            const float inv = length(ss);
            const int pos = tok_pos[t];
            T* row = key ? entry(t, pos) : q + (long long)t * d.q_cols() + hd * d.qh();
#pragma unroll
            for (int k = 0; k < NP; ++k)
                if (k * 32 + lane < end) store(row, pos, k * 32 + lane, turn(pos, k * 32 + lane, v[i][k], inv, g[k]));
        }
    } else {
        float ss = 0.0f;
        for (int pr = lane; 2 * pr < n; pr += 32) {
            const float2 v = pair(t0, pr, vec(bias, pr, 0.0f));
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, ss));
        }
        const float inv = length(ss);
        const int pos = tok_pos[t0];
        T* row = key ? entry(t0, pos) : q + (long long)t0 * d.q_cols() + hd * d.qh();
        for (int pr = lane; pr < end; pr += 32) store(row, pos, pr, turn(pos, pr, pair(t0, pr, vec(bias, pr, 0.0f)), inv, vec(gain, pr, 1.0f)));
    }
}

// ---- any sizes, f32 arithmetic throughout: one CTA per (token, head) ----------------------------------------------
template <typename T>
__global__ void __launch_bounds__(128) attn_paged_simt_kernel(const T* __restrict__ q, AttnDims d, const float* __restrict__ sink, const T* __restrict__ pool,
                                                              const int32_t* __restrict__ block_table, int max_pages,
                                                              const int32_t* __restrict__ tok_row, const int32_t* __restrict__ tok_pos,
                                                              const float* __restrict__ gate, T* __restrict__ out, int t_first) {
    extern __shared__ float sm[];
    float* qs = sm;                // [dim]
    float* o = qs + pad8(d.dim);   // [vdim]
    float* s = o + pad8(d.vdim);   // [128]
    float* red = s + 128;          // [8]
    chain_trigger();
    chain_wait();
    const int t = t_first + blockIdx.x, h = blockIdx.y, g = h / (d.H / d.G), warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    for (int i = threadIdx.x; i < d.dim; i += 128) qs[i] = to_f32(q[(long long)t * d.q_cols() + h * d.qh() + i]);
    for (int i = threadIdx.x; i < d.vdim; i += 128) o[i] = 0.0f;
    const int pos = tok_pos[t], k0 = d.mask.first(pos);
    const int32_t* bt = block_table + (long long)tok_row[t] * max_pages;
    float m = sink ? sink[h] : -INFINITY, l = sink ? 1.0f : 0.0f;
    for (int c0 = k0; c0 <= pos; c0 += 128) {
        const int n = min(128, pos + 1 - c0);
        __syncthreads();
        for (int j = warp; j < n; j += 4) {
            const int kp = c0 + j;
            float acc = 0.0f;
            for (int i = lane; i < d.dim; i += 32) acc = fmaf(qs[i], to_f32(*cache_at(pool, d, bt[kp / PAGE], g, 0, kp % PAGE, i)), acc);
            acc = warp_sum(acc);
            if (lane == 0) s[j] = acc * d.scale;
        }
        __syncthreads();
        const float v = threadIdx.x < n ? s[threadIdx.x] : -INFINITY;
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
        for (int i = threadIdx.x; i < d.vdim; i += 128) {
            float acc = o[i] * alpha;
            for (int j = 0; j < n; ++j) {
                const int kp = c0 + j;
                acc = fmaf(s[j], to_f32(*cache_at(pool, d, bt[kp / PAGE], g, 1, kp % PAGE, i)), acc);
            }
            o[i] = acc;
        }
    }
    const float f = (gate ? gate[(long long)t * d.H + h] : 1.0f) / l;
    for (int i = threadIdx.x; i < d.vdim; i += 128) out[(long long)t * d.out_cols() + h * d.vdim + i] = from_f32<T>(o[i] * f);
}

// ---- bf16 on the tensor cores -------------------------------------------------------------------------------------
// A CTA owns 8 NB (token, head of the group) rows of one segment and kv head, and a run of pages.  A producer thread fetches
// one block - the keys and values of the kv head in a page - per stage of a three-stage ring.  Each of four warps takes 16
// keys of the page: S^T[16 keys x rows] = K . Q^T with the keys as the 16-row operand, softmax along the keys with three
// shuffles per pair of rows, P^T from accumulator to operand layout by movmatrix, O^T[values x rows] += V^T . P^T.  The
// warps' partial sums are merged at the end; with several splits the CTA that arrives last merges theirs.  Scores, maxima and
// sums are fp32 (log2 domain), the weights enter the sum as bf16.  Waits for copies are bounded.
constexpr int AM_STAGES = 3;
constexpr int AM_WARPS = 4;
constexpr int AM_THREADS = (AM_WARPS + 1) * 32;
constexpr int AM_MAX_SPLITS = 64;
__host__ __device__ constexpr int am_pitch(int vp) { return vp + 4; }  // a row of partial sums: the columns, its maximum, its sum
constexpr int AM_ERR_FULL = 61, AM_ERR_EMPTY = 62;

struct AttnArgs {
    const __nv_bfloat16 *q, *pool;
    const int32_t *block_table, *seg_start, *seg_len, *seg_pos0, *seg_row, *tile_seg, *tile_r0;
    const float *gate, *sink;
    __nv_bfloat16* out;
    float* part;
    int *counters, *err;
    int max_pages, splits;
    float scale_log2;
};
static int am_vp(const AttnDims& d) { return d.vs() <= 2 ? d.vs() * 64 : 256; }  // value columns of the instance
static size_t am_smem(const AttnDims& d, int nb) {
    const size_t ring = (size_t)AM_STAGES * (d.ks() + d.vs()) * SLAB * 2, merge = (size_t)AM_WARPS * 8 * nb * am_vp(d) * 4;
    return std::max(ring, merge) + 1024 + (size_t)8 * nb * (d.ks() * 64 + 8) * 2;
}

__device__ __forceinline__ uint32_t movmatrix_t(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

template <int NB, int VT>  // VT: 16-wide tiles of the values
__global__ void __launch_bounds__(AM_THREADS, 1) attn_paged_mma_kernel(AttnArgs a, AttnDims d) {
    constexpr int R = 8 * NB, VP = VT * 16;
    extern __shared__ uint8_t am_dyn[];
    uint8_t* ring = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(am_dyn) + 1023) & ~uintptr_t(1023));
    __shared__ __align__(8) uint64_t full_bar[AM_STAGES], empty_bar[AM_STAGES];
    __shared__ int abort_flag, is_last;
    __shared__ float sm_m[AM_WARPS][R], sm_l[AM_WARPS][R];
    chain_trigger();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int ks = d.ks(), stage_bytes = (ks + d.vs()) * SLAB * 2, qp = ks * 64 + 8, gs = d.H / d.G;
    const int ring_bytes = max(AM_STAGES * stage_bytes, AM_WARPS * R * VP * 4);
    __nv_bfloat16* qs = reinterpret_cast<__nv_bfloat16*>(ring + ring_bytes);  // [R][qp]
    if (threadIdx.x == 0) {
        for (int s = 0; s < AM_STAGES; ++s) {
            tc::mbar_init(&full_bar[s], 1);
            tc::mbar_init(&empty_bar[s], AM_WARPS);
        }
        abort_flag = 0;
        tc::mbar_fence_init();
    }
    __syncthreads();
    chain_wait();
    const int tile = blockIdx.x, g = blockIdx.y, sp = blockIdx.z;
    const int seg = a.tile_seg[tile], r0 = a.tile_r0[tile];
    const int start = a.seg_start[seg], pos0 = a.seg_pos0[seg];
    const int n_rows = min(R, a.seg_len[seg] * gs - r0);
    const int key_lo = d.mask.first(pos0 + r0 / gs), key_hi = pos0 + (r0 + n_rows - 1) / gs + 1;
    const int pg_lo = key_lo / PAGE, n_pg = (key_hi - 1) / PAGE - pg_lo + 1;
    const int live = min(a.splits, n_pg);  // the grid is made for the longest context
    if (sp >= live) return;
    const int pb = pg_lo + n_pg * sp / live, n_it = pg_lo + n_pg * (sp + 1) / live - pb;
    const int32_t* bt = a.block_table + (long long)a.seg_row[seg] * a.max_pages + pb;

    // queries (columns behind the head's are zero)
    for (int i = threadIdx.x; i < R * ks * 8; i += AM_THREADS) {
        const int r = i / (ks * 8), c = (i - r * ks * 8) * 8, row = r0 + r;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < n_rows && c < d.qh())
            v = *reinterpret_cast<const uint4*>(a.q + (long long)(start + row / gs) * d.q_cols() + (g * gs + row % gs) * d.qh() + c);
        *reinterpret_cast<uint4*>(qs + r * qp + c) = v;
    }
    __syncthreads();

    float m[NB][2], l[NB][2], o[VT][NB][4];
#pragma unroll
    for (int b = 0; b < NB; ++b) {
        m[b][0] = m[b][1] = -INFINITY;
        l[b][0] = l[b][1] = 0.0f;
#pragma unroll
        for (int j = 0; j < VT; ++j) o[j][b][0] = o[j][b][1] = o[j][b][2] = o[j][b][3] = 0.0f;
    }
    if (warp == AM_WARPS) {
        if (lane == 0) {
            int issued = 0;
            for (int it = 0; it < n_it; ++it) {
                const int s = it % AM_STAGES;
                if (it >= AM_STAGES && !tc::mbar_wait(&empty_bar[s], ((it / AM_STAGES) - 1) & 1, &abort_flag, a.err, AM_ERR_EMPTY)) break;
                tc::mbar_expect_tx(&full_bar[s], stage_bytes);
                tc::bulk_load(ring + s * stage_bytes, a.pool + (long long)(bt[it] * d.G + g) * (stage_bytes / 2), stage_bytes, &full_bar[s]);
                issued = it + 1;
            }
            if (abort_flag) {  // let the copies in flight land (bounded)
                const long long t0 = clock64();
                for (int it = max(0, issued - AM_STAGES); it < issued; ++it)
                    while (!tc::mbar_try_wait(&full_bar[it % AM_STAGES], (it / AM_STAGES) & 1) && clock64() - t0 < tc::WAIT_LIMIT_CYCLES) {}
            }
        }
    } else {
        int hi[NB][2], lo[NB][2];  // keys [lo, hi] of this lane's rows
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = b * 8 + (lane & 3) * 2 + e, p = pos0 + (r0 + r) / gs;
                hi[b][e] = r < n_rows ? p : -1;
                lo[b][e] = d.mask.first(p);
            }
        const int mi = lane >> 3, mr = lane & 7;
        const int krow = warp * 16 + (mi & 1) * 8 + mr, kchunk = mi >> 1;  // keys: matrices 0 / 1 = keys 0-7 / 8-15, 2 / 3 = 8 columns on
        const int vrow = warp * 16 + (mi >> 1) * 8 + mr, vchunk = mi & 1;  // values (transposed): 0 / 1 = columns, 2 / 3 = keys 8-15
        const uint32_t q_addr = smem_u32(qs + mr * qp + mi * 8);           // queries: matrices = four 8-column pieces of two steps
        for (int it = 0; it < n_it; ++it) {
            const int s = it % AM_STAGES;
            if (!tc::mbar_wait(&full_bar[s], (it / AM_STAGES) & 1, &abort_flag, a.err, AM_ERR_FULL)) break;
            const int key0 = (pb + it) * PAGE + warp * 16;
            if (key0 < key_hi && key0 + 16 > key_lo) {
                const uint32_t kbase = smem_u32(ring + s * stage_bytes), vbase = kbase + ks * SLAB * 2;
                float sc[NB][4];
#pragma unroll
                for (int b = 0; b < NB; ++b) sc[b][0] = sc[b][1] = sc[b][2] = sc[b][3] = 0.0f;
                for (int slab = 0; slab < ks; ++slab)
#pragma unroll
                    for (int k2 = 0; k2 < 2; ++k2) {  // two 16-wide steps
                        uint32_t a0[4], a1[4];
                        const int c0 = k2 * 4 + kchunk, c1 = c0 + 2;
                        ldsm_x4(kbase + slab * SLAB * 2 + krow * 128 + ((c0 ^ (krow & 7)) << 4), a0);
                        ldsm_x4(kbase + slab * SLAB * 2 + krow * 128 + ((c1 ^ (krow & 7)) << 4), a1);
#pragma unroll
                        for (int b = 0; b < NB; ++b) {
                            uint32_t qf[4];
                            ldsm_x4(q_addr + (b * 8 * qp + slab * 64 + k2 * 32) * 2, qf);
                            mma_16816(sc[b], a0, qf[0], qf[1]);
                            mma_16816(sc[b], a1, qf[2], qf[3]);
                        }
                    }
                const int k0 = key0 + (lane >> 2), k1 = k0 + 8;
                uint32_t pb0[NB], pb1[NB];
#pragma unroll
                for (int b = 0; b < NB; ++b) {
                    float x[4];
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        x[e] = k0 >= lo[b][e] && k0 <= hi[b][e] ? sc[b][e] * a.scale_log2 : -INFINITY;
                        x[2 + e] = k1 >= lo[b][e] && k1 <= hi[b][e] ? sc[b][2 + e] * a.scale_log2 : -INFINITY;
                    }
                    float mx[2] = {fmaxf(x[0], x[2]), fmaxf(x[1], x[3])}, corr[2];
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
#pragma unroll
                        for (int sh = 4; sh < 32; sh <<= 1) mx[e] = fmaxf(mx[e], __shfl_xor_sync(0xffffffffu, mx[e], sh));
                        const float mn = fmaxf(m[b][e], mx[e]), ref = mn == -INFINITY ? 0.0f : mn;
                        corr[e] = exp2f(m[b][e] - ref);
                        m[b][e] = mn;
                        x[e] = exp2f(x[e] - ref);
                        x[2 + e] = exp2f(x[2 + e] - ref);
                        l[b][e] = fmaf(l[b][e], corr[e], x[e] + x[2 + e]);
                    }
#pragma unroll
                    for (int j = 0; j < VT; ++j) {
                        o[j][b][0] *= corr[0]; o[j][b][1] *= corr[1];
                        o[j][b][2] *= corr[0]; o[j][b][3] *= corr[1];
                    }
                    pb0[b] = movmatrix_t(pack_bf16x2(x[0], x[1]));
                    pb1[b] = movmatrix_t(pack_bf16x2(x[2], x[3]));
                }
#pragma unroll
                for (int j = 0; j < VT; ++j) {
                    if (VT == 16 && j >= d.vs() * 4) break;
                    const int c = j * 2 + vchunk;
                    uint32_t v[4];
                    ldsm_x4_trans(vbase + (c >> 3) * SLAB * 2 + vrow * 128 + (((c & 7) ^ (vrow & 7)) << 4), v);
#pragma unroll
                    for (int b = 0; b < NB; ++b) mma_16816(o[j][b], v, pb0[b], pb1[b]);
                }
            }
            __syncwarp();
            if (lane == 0) tc::mbar_arrive(&empty_bar[s]);
        }
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int e = 0; e < 2; ++e)
#pragma unroll
                for (int sh = 4; sh < 32; sh <<= 1) l[b][e] += __shfl_xor_sync(0xffffffffu, l[b][e], sh);
    }
    __syncthreads();  // every stage has been consumed: the ring becomes the merge buffer [warp][row][column]
    if (abort_flag) return;
    float* sm_o = reinterpret_cast<float*>(ring);
    if (warp < AM_WARPS) {
        const int c = lane >> 2;
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int r = b * 8 + (lane & 3) * 2;
#pragma unroll
            for (int j = 0; j < VT; ++j) {
                float* dst = sm_o + (warp * R + r) * VP + j * 16 + c;
                dst[0] = o[j][b][0];
                dst[VP] = o[j][b][1];
                dst[8] = o[j][b][2];
                dst[VP + 8] = o[j][b][3];
            }
            if (c == 0) {
                sm_m[warp][r] = m[b][0]; sm_m[warp][r + 1] = m[b][1];
                sm_l[warp][r] = l[b][0]; sm_l[warp][r + 1] = l[b][1];
            }
        }
    }
    __syncthreads();
    // the sink joins the denominator once, at the very end
    auto finish = [&](int r, int c, float acc, float L, float M) {
        const int row = r0 + r, t = start + row / gs, h = g * gs + row % gs;
        const float s2 = a.sink ? a.sink[h] * LOG2E : -INFINITY, top = fmaxf(M, s2), f = exp2f(M - top);
        const float gv = a.gate ? a.gate[(long long)t * d.H + h] : 1.0f;
        a.out[(long long)t * d.out_cols() + h * d.vdim + c] = __float2bfloat16_rn(acc * f / fmaf(L, f, exp2f(s2 - top)) * gv);
    };
    float* part = a.part + (long long)(tile * d.G + g) * a.splits * R * am_pitch(VP);
    for (int e = threadIdx.x; e < n_rows * VP; e += AM_THREADS) {
        const int r = e / VP, c = e % VP;
        if (live == 1 && c >= d.vdim) continue;
        float M = -INFINITY, acc = 0.0f, L = 0.0f;
#pragma unroll
        for (int w = 0; w < AM_WARPS; ++w) M = fmaxf(M, sm_m[w][r]);
#pragma unroll
        for (int w = 0; w < AM_WARPS; ++w) {
            const float f = sm_m[w][r] == -INFINITY ? 0.0f : exp2f(sm_m[w][r] - M);
            acc = fmaf(f, sm_o[(w * R + r) * VP + c], acc);
            L = fmaf(f, sm_l[w][r], L);
        }
        if (live == 1) {
            finish(r, c, acc, L, M);
        } else {
            float* dst = part + ((long long)sp * R + r) * am_pitch(VP);
            dst[c] = acc;
            if (c == 0) { dst[VP] = M; dst[VP + 1] = L; }
        }
    }
    if (live == 1) return;
    __syncthreads();  // all partial stores of the CTA precede the release below
    if (threadIdx.x == 0) {
        int old;
        int* ctr = a.counters + tile * d.G + g;
        asm volatile("atom.add.acq_rel.gpu.global.s32 %0, [%1], 1;" : "=r"(old) : "l"(ctr) : "memory");
        is_last = old == live - 1;
        if (is_last) *ctr = 0;  // ready for the next launch
    }
    __syncthreads();
    if (!is_last) return;
    // weight of every split's partial sum per row, then four columns per thread
    const long long stride = (long long)R * am_pitch(VP);
    float* wts = reinterpret_cast<float*>(ring);  // [R][AM_MAX_SPLITS]
    for (int r = warp; r < n_rows; r += AM_WARPS + 1) {
        float ms[2], ls[2];
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            const float* src = part + (long long)(lane + 32 * i) * stride + r * am_pitch(VP) + VP;
            const bool on = lane + 32 * i < live;
            ms[i] = on ? __ldcg(src) : -INFINITY;
            ls[i] = on ? __ldcg(src + 1) : 0.0f;
        }
        const float M = warp_max(fmaxf(ms[0], ms[1])), f0 = exp2f(ms[0] - M), f1 = exp2f(ms[1] - M);  // (M is finite: a row sees its own key)
        const float L = warp_sum(fmaf(f0, ls[0], f1 * ls[1]));
        wts[r * AM_MAX_SPLITS + lane] = f0;
        wts[r * AM_MAX_SPLITS + lane + 32] = f1;
        if (lane == 0) { sm_m[0][r] = M; sm_l[0][r] = L; }
    }
    __syncthreads();
    for (int e = threadIdx.x; e < n_rows * (VP / 4); e += AM_THREADS) {
        const int r = e / (VP / 4), c = e % (VP / 4) * 4;
        const float* src = part + r * am_pitch(VP) + c;
        float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int s = 0; s < live; ++s) {
            const float4 v = __ldcg(reinterpret_cast<const float4*>(src + s * stride));
            const float f = wts[r * AM_MAX_SPLITS + s];
            acc.x = fmaf(f, v.x, acc.x); acc.y = fmaf(f, v.y, acc.y); acc.z = fmaf(f, v.z, acc.z); acc.w = fmaf(f, v.w, acc.w);
        }
        const float o4[4] = {acc.x, acc.y, acc.z, acc.w};
#pragma unroll
        for (int i = 0; i < 4; ++i)
            if (c + i < d.vdim) finish(r, c + i, o4[i], sm_l[0][r], sm_m[0][r]);
    }
}

// ---- launches -----------------------------------------------------------------------------------------------------
template <typename T>
static jsm_status prep_typed(const float* wide, const AttnDims& d, const AttnWeights& w, float eps, const AttnCache& cache, bool own_kv, const StepTokens& tk,
                             void* q, float* gate, cudaStream_t st) {
    const int units = d.H + (own_kv ? 2 * d.G : 0) + (d.gated ? 1 : 0);
    auto go = [&](auto kernel, int tok) {
        return launch_chained(kernel, dim3((tk.T + tok - 1) / tok, (units + 7) / 8), dim3(256), 0, st, wide, d, w, eps, (T*)cache.pool, cache.block_table,
                              cache.max_pages, cache.rope, tk.tok_row, tk.tok_pos, own_kv ? 1 : 0, tk.T, (T*)q, gate);
    };
    const bool many = tk.T >= 512;
    JSM_CUDA_CHECK(d.ks() == 1 ? many ? go(attn_prep_kernel<T, 1, 4>, 4) : go(attn_prep_kernel<T, 1, 1>, 1)
                   : d.ks() == 2 ? many ? go(attn_prep_kernel<T, 2, 4>, 4) : go(attn_prep_kernel<T, 2, 1>, 1) : go(attn_prep_kernel<T, 0, 1>, 1));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
jsm_status attn_prep_launch(bool f32, const float* wide, const AttnDims& d, const AttnWeights& w, float eps, const AttnCache& cache, bool own_kv,
                            const StepTokens& tk, void* q, float* gate, cudaStream_t st) {
    return f32 ? prep_typed<float>(wide, d, w, eps, cache, own_kv, tk, q, gate, st) : prep_typed<__nv_bfloat16>(wide, d, w, eps, cache, own_kv, tk, q, gate, st);
}

bool attn_mma_usable(const AttnDims& d) { return d.ks() <= 4 && d.vs() <= 4; }
int attn_tile_rows(const AttnDims& d, bool decode) { return decode && d.H / d.G <= 8 ? 8 : d.vs() <= 2 ? 32 : 16; }
static int attn_splits(const AttnDims& d, int n_tiles, int max_keys) {
    const int pages = max_keys / PAGE + 2, ctas = std::max(1, n_tiles * d.G);
    return std::max(1, std::min({2 * sm_count() / ctas, pages / 2, AM_MAX_SPLITS}));
}
size_t attn_part_floats(const AttnDims& d) { return (size_t)2 * sm_count() * 32 * am_pitch(am_vp(d)); }
int attn_counters() { return 2 * sm_count(); }

template <int NB, int VT>
static jsm_status launch_attn_mma(const AttnArgs& a, const AttnDims& d, int n_tiles, cudaStream_t st) {
    static bool attr_done = false;
    if (!attr_done) {
        JSM_CUDA_CHECK(cudaFuncSetAttribute(attn_paged_mma_kernel<NB, VT>, cudaFuncAttributeMaxDynamicSharedMemorySize, 224 * 1024));
        attr_done = true;
    }
    JSM_CUDA_CHECK(launch_chained(attn_paged_mma_kernel<NB, VT>, dim3(n_tiles, d.G, a.splits), dim3(AM_THREADS), am_smem(d, NB), st, a, d));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

jsm_status attn_paged_launch(bool f32, const AttnDims& d, const AttnWeights& w, const AttnCache& cache, const StepTokens& tk, const AttnTiles& tl,
                             const void* q, const float* gate, const AttnScratch& sc, void* out, cudaStream_t st) {
    if (tl.n_tiles <= 0 || tl.t_count <= 0) return JSM_OK;
    const float* gates = d.gated ? gate : nullptr;
    if (f32 || !attn_mma_usable(d)) {
        const size_t smem = sizeof(float) * (pad8(d.dim) + pad8(d.vdim) + 128 + 8);
        if (smem > 48 * 1024) JSM_FAIL(JSM_UNSUPPORTED, "attention: heads of %d / %d components", d.dim, d.vdim);
        if (f32)
            JSM_CUDA_CHECK(launch_chained(attn_paged_simt_kernel<float>, dim3(tl.t_count, d.H), dim3(128), smem, st, (const float*)q, d, w.sink,
                                          (const float*)cache.pool, cache.block_table, cache.max_pages, tk.tok_row, tk.tok_pos, gates, (float*)out,
                                          tl.t_first));
        else
            JSM_CUDA_CHECK(launch_chained(attn_paged_simt_kernel<__nv_bfloat16>, dim3(tl.t_count, d.H), dim3(128), smem, st, (const __nv_bfloat16*)q, d,
                                          w.sink, (const __nv_bfloat16*)cache.pool, cache.block_table, cache.max_pages, tk.tok_row, tk.tok_pos, gates,
                                          (__nv_bfloat16*)out, tl.t_first));
        JSM_LAUNCH_CHECK();
        return JSM_OK;
    }
    AttnArgs a;
    a.q = (const __nv_bfloat16*)q; a.pool = (const __nv_bfloat16*)cache.pool; a.block_table = cache.block_table;
    a.seg_start = tk.seg_start; a.seg_len = tk.seg_len; a.seg_pos0 = tk.seg_pos0; a.seg_row = tk.seg_row;
    a.tile_seg = tl.tile_seg; a.tile_r0 = tl.tile_r0;
    a.gate = gates; a.sink = w.sink; a.out = (__nv_bfloat16*)out; a.part = sc.part; a.counters = sc.counters; a.err = tc_error_word();
    a.max_pages = cache.max_pages;
    a.splits = attn_splits(d, tl.n_tiles, tl.max_keys);
    a.scale_log2 = d.scale * LOG2E;
    if (a.splits > 1 && ((size_t)tl.n_tiles * d.G * a.splits * tl.rows * am_pitch(am_vp(d)) > sc.part_floats || tl.n_tiles * d.G > sc.n_counters))
        JSM_FAIL(JSM_INVALID_ARG, "attention: workspace of %zu floats for %d tiles x %d heads in %d splits", sc.part_floats, tl.n_tiles, d.G, a.splits);
    const int vs = d.vs();
    if (tl.rows == 8) return vs == 1 ? launch_attn_mma<1, 4>(a, d, tl.n_tiles, st) : vs == 2 ? launch_attn_mma<1, 8>(a, d, tl.n_tiles, st)
                                                                                          : launch_attn_mma<1, 16>(a, d, tl.n_tiles, st);
    return vs == 1 ? launch_attn_mma<4, 4>(a, d, tl.n_tiles, st) : vs == 2 ? launch_attn_mma<4, 8>(a, d, tl.n_tiles, st)
                                                                         : launch_attn_mma<2, 16>(a, d, tl.n_tiles, st);
}

}  // namespace jsm
