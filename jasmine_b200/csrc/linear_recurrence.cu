// Linear recurrences with a matrix state per head, over segments of consecutive tokens of many sequences:
//
//   decayed sum  S <- g S + k v^T                               g: a constant of the head
//   delta rule   S <- g S;  S <- S + k u^T, u = beta (v - S^T k)   g = exp(-exp(A) softplus(a + dt)), beta = sigmoid(b) per token
//   both         o = S^T q
//
// q, k and v have passed the short convolution (short_conv_launch; one tap of weight 1 where a design has none) and its
// silu; the delta rule makes unit vectors of q and k per head first, x / sqrt(sum(x^2) + 1e-6), and q also dk^(-1/2).  The
// state and all of this arithmetic is fp32; q, k, v, o and the gates z are activations (bf16 or f32).  A sequence's state lives
// in a slot; a segment that starts at position 0 starts from zeros whatever the slot holds.
//
// Prompts of bf16 models run on the tensor cores in chunks of 64 tokens (rec_chunk_prep, rec_chunk): with G the running sum of
// log g in the chunk and S0 the state before it,
//     (I + A) U = diag(beta) (V - diag(e^G) K S0),   A[t][j] = beta_t e^(G_t - G_j) (k_t . k_j), j < t   (decayed sum: U = V)
//     O = diag(e^G) Q S0 + P U,                      P[t][j] = e^(G_t - G_j) (q_t . k_j), j <= t
//     S = e^(G_end) S0 + sum_j e^(G_end - G_j) k_j u_j^T.
// f32 models and heads of more than 128 key components walk the tokens one by one (rec_scan), as does a decode step (rec_step).
//
// Row of the input projection: [q: G heads | k: G heads | v: H heads | z: H heads], heads at pitches padded to 8; head h uses
// query / key head h / (H / G).  State: [slot][head][kp][vp].
#include "decoder_ops.cuh"
#include "mma_utils.cuh"
#include "tc_utils.cuh"
#include <math.h>
#include <algorithm>

namespace jsm {

using tc::smem_u32;

constexpr float UNIT_EPS = 1e-6f;

struct RecArgs {
    const void *qkv, *z, *x, *ba_w;   // qkv: act [T][conv cols]; z: first gate column of the input projection, pitch raw
    const float *ba, *A, *dt_bias, *decay, *log_decay, *norm;
    float* S;
    void* out;
    const int32_t *seg_start, *seg_len, *seg_pos0, *seg_slot;
    float eps, q_scale;
    int x_pitch;
};

__device__ __forceinline__ float rec_sigmoid(float x) { return 1.0f / (1.0f + expf(-x)); }
__device__ __forceinline__ float rec_softplus(float x) { return x > 20.0f ? x : log1pf(expf(x)); }

// ---- prompts, any sizes up to 256 key components, f32 arithmetic throughout ---------------------------------------
// A CTA owns 16 columns of one head's state; eight threads share a column (rows sub, sub + 8, ...).
constexpr int RS_COLS = 16, RS_SUB = 8, RS_THREADS = RS_COLS * RS_SUB, RS_TT = 16;

template <typename T, int NS, bool DELTA>
__global__ void __launch_bounds__(RS_THREADS) rec_scan_kernel(RecArgs a, RecDims d) {
    constexpr int KW = 8 * NS;  // rows of the state, rounded up
    __shared__ float ks[RS_TT][KW], qs[RS_TT][KW], vs[RS_TT][RS_COLS], gs[RS_TT], bs[RS_TT];
    chain_trigger();
    chain_wait();
    const int tid = threadIdx.x, col = tid / RS_SUB, sub = tid % RS_SUB, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, g = h / (d.H / d.G), seg = blockIdx.z, kp = d.kp(), vp = d.vp(), cc = d.conv_cols();
    const int c = blockIdx.x * RS_COLS + col;
    const bool live = c < vp;
    const int start = a.seg_start[seg], len = a.seg_len[seg];
    float* state = a.S + ((long long)a.seg_slot[seg] * d.H + h) * kp * vp + c;
    const bool fresh = a.seg_pos0[seg] == 0;
    float S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int r = sub + 8 * i;
        S[i] = live && r < kp && !fresh ? state[(long long)r * vp] : 0.0f;
    }
    const T* qkv = static_cast<const T*>(a.qkv);
    const float decay = DELTA ? 0.0f : a.decay[h];
    for (int t0 = 0; t0 < len; t0 += RS_TT) {
        const int n = min(RS_TT, len - t0);
        __syncthreads();
        for (int t = warp; t < n; t += RS_THREADS / 32) {
            const T* row = qkv + (long long)(start + t0 + t) * cc;
            float sq = 0.0f, sk = 0.0f;
            for (int i = lane; i < KW; i += 32) {
                const float q = i < kp ? to_f32(row[g * kp + i]) : 0.0f, k = i < kp ? to_f32(row[(d.G + g) * kp + i]) : 0.0f;
                qs[t][i] = q; ks[t][i] = k;
                sq = fmaf(q, q, sq); sk = fmaf(k, k, sk);
            }
            if (DELTA) {
                sq = sqrtf(warp_sum(sq) + UNIT_EPS);
                sk = sqrtf(warp_sum(sk) + UNIT_EPS);
                for (int i = lane; i < KW; i += 32) { qs[t][i] = qs[t][i] / sq * a.q_scale; ks[t][i] /= sk; }
            }
            const int vc = blockIdx.x * RS_COLS + lane;
            if (lane < RS_COLS) vs[t][lane] = vc < vp ? to_f32(row[2 * d.G * kp + h * vp + vc]) : 0.0f;
            if (DELTA && lane == 0) {
                const float* ba = a.ba + (long long)(start + t0 + t) * d.ba_cols();
                bs[t] = rec_sigmoid(ba[h]);
                gs[t] = expf(a.A[h] * rec_softplus(ba[d.ba_cols() / 2 + h] + a.dt_bias[h]));
            }
        }
        __syncthreads();
        for (int t = 0; t < n; ++t) {
            const float gt = DELTA ? gs[t] : decay;
            float u = vs[t][col], k[NS], o = 0.0f;
#pragma unroll
            for (int i = 0; i < NS; ++i) { k[i] = ks[t][sub + 8 * i]; S[i] *= gt; }
            if (DELTA) {
                float p = 0.0f;
#pragma unroll
                for (int i = 0; i < NS; ++i) p = fmaf(S[i], k[i], p);
#pragma unroll
                for (int x = 1; x < RS_SUB; x <<= 1) p += __shfl_xor_sync(0xffffffffu, p, x);
                u = bs[t] * (u - p);
            }
#pragma unroll
            for (int i = 0; i < NS; ++i) {
                S[i] = fmaf(k[i], u, S[i]);
                o = fmaf(S[i], qs[t][sub + 8 * i], o);
            }
#pragma unroll
            for (int x = 1; x < RS_SUB; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
            if (live && sub == 0) static_cast<T*>(a.out)[(long long)(start + t0 + t) * d.H * vp + h * vp + c] = from_f32<T>(o);
        }
    }
    if (live)
#pragma unroll
        for (int i = 0; i < NS; ++i)
            if (sub + 8 * i < kp) state[(long long)(sub + 8 * i) * vp] = S[i];
}

// ---- prompts on the tensor cores ----------------------------------------------------------------------------------
// The matrix operands are the bf16 activations themselves: unit norms, decays and beta are fp32 factors per token around the
// products.  fp32 operands (the state, U and its right-hand side, the inverse of I + A) enter as a sum of two bf16 numbers, so
// that what feeds the state keeps 16 bits; P enters as bf16, as attention weights do.
constexpr int RC_C = REC_CHUNK;       // tokens per chunk
constexpr int RC_P = RC_C + 8;        // pitch of a chunk matrix (bf16)
constexpr int RC_MAT = RC_C * RC_P * 2;
constexpr int RC_SCAL = 4 * RC_C * 4 + 16;  // per token: factors of v, K S0, Q S0 and k u^T; the chunk's decay
constexpr int RC_SLAB = RC_C * 128;   // bytes of 64 key components of a chunk
constexpr int RC_ERR_FULL = 71;
constexpr float LOG_MIN = -120.0f;    // e^-120 is 0 in fp32
__host__ __device__ inline int rc_block(bool delta) { return (delta ? 3 : 1) * RC_MAT + RC_SCAL; }  // bytes per (chunk, head): [T hi | T lo |] P | factors

__host__ __device__ inline int rc_prep_tiles(int kw, bool delta) {  // bytes of the tiles of K and Q, and of the inverse behind them
    const int tiles = 2 * RC_C * (kw + 8) * 2, x = delta ? RC_C * 68 * 4 : 0;
    return tiles > x ? tiles : x;
}

__host__ __device__ inline int rc_stage(int tile, int cols, bool delta) { return (2 * tile + RC_C * cols * 2 + rc_block(delta) + 1023) & ~1023; }
// Per (chunk, head): the factors, P, and the inverse T of I + A.  Eight warps.
template <bool DELTA>
__global__ void __launch_bounds__(256) rec_chunk_prep_kernel(RecArgs a, RecDims d, const int32_t* __restrict__ chunk_seg, const int32_t* __restrict__ chunk_t0,
                                                             uint8_t* __restrict__ ws, int kw) {
    extern __shared__ __align__(16) uint8_t rc_dyn[];
    const int pitch = kw + 8;  // kw: key components rounded up to 16
    __nv_bfloat16* ks = reinterpret_cast<__nv_bfloat16*>(rc_dyn);          // [64][pitch]
    __nv_bfloat16* qs = ks + RC_C * pitch;                                 // [64][pitch]
    float* As = reinterpret_cast<float*>(rc_dyn + rc_prep_tiles(kw, DELTA));  // [64][68], strictly lower
    float* Xs = reinterpret_cast<float*>(rc_dyn);                          // [64][68]: the inverse, where the tiles were
    __shared__ float G[RC_C], rk[RC_C], rq[RC_C], beta[RC_C], half_sum;
    chain_trigger();
    chain_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int seg = chunk_seg[blockIdx.x], t0 = chunk_t0[blockIdx.x], h = blockIdx.y, g = h / (d.H / d.G);
    const int n = min(RC_C, a.seg_len[seg] - t0), kp = d.kp(), vec = kw / 8;
    const long long first = a.seg_start[seg] + t0;
    const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(a.qkv) + first * d.conv_cols() + g * kp;
    for (int i = tid; i < RC_C * vec; i += 256) {
        const int r = i / vec, c = (i - r * vec) * 8;
        uint4 k = make_uint4(0, 0, 0, 0), q = k;
        if (r < n && c < kp) {
            const __nv_bfloat16* row = qkv + (long long)r * d.conv_cols() + c;
            q = *reinterpret_cast<const uint4*>(row);
            k = *reinterpret_cast<const uint4*>(row + d.G * kp);
        }
        *reinterpret_cast<uint4*>(ks + r * pitch + c) = k;
        *reinterpret_cast<uint4*>(qs + r * pitch + c) = q;
    }
    // running sum of the log decays
    if (tid < RC_C) {
        float lg = 0.0f, b = 0.0f;
        if (tid < n) {
            if (DELTA) {
                const float* ba = a.ba + (first + tid) * d.ba_cols();
                b = rec_sigmoid(ba[h]);
                lg = fmaxf(a.A[h] * rec_softplus(ba[d.ba_cols() / 2 + h] + a.dt_bias[h]), LOG_MIN);
            } else {
                lg = fmaxf(a.log_decay[h], LOG_MIN);
            }
        }
        beta[tid] = b;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float v = __shfl_up_sync(0xffffffffu, lg, o);
            if (lane >= o) lg += v;
        }
        G[tid] = lg;
        if (tid == 31) half_sum = lg;
    }
    __syncthreads();
    if (tid >= 32 && tid < RC_C) G[tid] += half_sum;
    if (DELTA) {  // lengths: four threads per row of k, then of q
        for (int m = 0; m < 2; ++m) {
            const __nv_bfloat16* row = (m ? qs : ks) + (tid >> 2) * pitch;
            float ss = 0.0f;
            for (int c = (tid & 3) * 8; c < kw; c += 32) {
                float v[8];
                load_f32x8(row + c, v);
#pragma unroll
                for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
            }
            ss += __shfl_xor_sync(0xffffffffu, ss, 1);
            ss += __shfl_xor_sync(0xffffffffu, ss, 2);
            if ((tid & 3) == 0) (m ? rq : rk)[tid >> 2] = (m ? a.q_scale : 1.0f) / sqrtf(ss + UNIT_EPS);
        }
    } else if (tid < RC_C) {
        rk[tid] = rq[tid] = 1.0f;
    }
    __syncthreads();
    uint8_t* out = ws + ((long long)blockIdx.x * d.H + h) * rc_block(DELTA);
    __nv_bfloat16* Pm = reinterpret_cast<__nv_bfloat16*>(out + (DELTA ? 2 * RC_MAT : 0));
    // products with the keys: warps 0-3 k . k (16 rows each), warps 4-7 q . k
    if (DELTA || warp >= 4) {
        const bool is_q = warp >= 4;
        const int mt = warp & 3, lm = lane >> 3, lr = lane & 7;
        float acc[8][4];
#pragma unroll
        for (int j = 0; j < 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.0f;
        const uint32_t a_addr = smem_u32((is_q ? qs : ks) + (mt * 16 + (lm & 1) * 8 + lr) * pitch + (lm >> 1) * 8);
        const uint32_t b_addr = smem_u32(ks + ((lm >> 1) * 8 + lr) * pitch + (lm & 1) * 8);
        for (int k = 0; k < kw; k += 16) {
            uint32_t af[4];
            ldsm_x4(a_addr + k * 2, af);
#pragma unroll
            for (int jp = 0; jp < 4; ++jp) {
                if (jp > mt) break;
                uint32_t bf[4];
                ldsm_x4(b_addr + (jp * 16 * pitch + k) * 2, bf);
                mma_16816(acc[2 * jp], af, bf[0], bf[1]);
                mma_16816(acc[2 * jp + 1], af, bf[2], bf[3]);
            }
        }
#pragma unroll
        for (int j = 0; j < 8; ++j)
#pragma unroll
            for (int e = 0; e < 4; e += 2) {
                const int t = mt * 16 + (lane >> 2) + (e >> 1) * 8, c = j * 8 + (lane & 3) * 2;
                float v[2];
#pragma unroll
                for (int x = 0; x < 2; ++x) {
                    const bool on = is_q ? c + x <= t : c + x < t;
                    v[x] = on ? acc[j][e + x] * rk[c + x] * (is_q ? rq[t] : beta[t] * rk[t]) * expf(G[t] - G[c + x]) : 0.0f;
                }
                if (is_q) *reinterpret_cast<uint32_t*>(Pm + t * RC_P + c) = pack_bf16x2(v[0], v[1]);
                else *reinterpret_cast<float2*>(As + t * 68 + c) = make_float2(v[0], v[1]);
            }
    }
    if (tid < RC_C) {
        float* f = reinterpret_cast<float*>(out + (DELTA ? 3 : 1) * RC_MAT);
        const bool on = tid < n;
        const float e = expf(G[tid]), last = G[RC_C - 1];
        f[tid] = !on ? 0.0f : DELTA ? beta[tid] : 1.0f;
        f[RC_C + tid] = on ? beta[tid] * e * rk[tid] : 0.0f;
        f[2 * RC_C + tid] = on ? e * rq[tid] : 0.0f;
        f[3 * RC_C + tid] = on ? expf(last - G[tid]) * rk[tid] : 0.0f;
        if (tid == 0) f[4 * RC_C] = expf(last);
    }
    if (!DELTA) return;
    __syncthreads();
    // The inverse X of I + A in blocks: 16 x 16 diagonal blocks by forward substitution (a thread per column), then twice
    //     [[D1, 0], [A21, D2]]^-1 = [[X1, 0], [-X2 A21 X1, X2]].
    // The products A21 X1 rest in the upper triangle of As, which nothing else uses.
    for (int i = tid; i < RC_C * 64; i += 256) {
        const int r = i >> 6, c = i & 63;
        if (r >> 4 < c >> 4) Xs[r * 68 + c] = 0.0f;
    }
    if (tid < RC_C) {
        const int b = tid & 48, j = tid & 15;
        float x[16];
#pragma unroll
        for (int t = 0; t < 16; ++t) {
            float sum = 0.0f;
#pragma unroll
            for (int i = 0; i < t; i += 4) {  // (entries of the row from t on are zero)
                const float4 r = *reinterpret_cast<const float4*>(As + (b + t) * 68 + b + i);
                sum = fmaf(r.x, x[i], sum);
                if (i + 1 < t) sum = fmaf(r.y, x[i + 1], sum);
                if (i + 2 < t) sum = fmaf(r.z, x[i + 2], sum);
                if (i + 3 < t) sum = fmaf(r.w, x[i + 3], sum);
            }
            x[t] = (t == j ? 1.0f : 0.0f) - sum;
            Xs[(b + t) * 68 + b + j] = x[t];
        }
    }
    __syncthreads();
    {
        const int m = (tid >> 7) * 32, r = (tid & 127) >> 3, c = (tid & 7) * 2;
        float y0 = 0.0f, y1 = 0.0f;
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float v = As[(m + 16 + r) * 68 + m + k];
            const float2 x = *reinterpret_cast<const float2*>(Xs + (m + k) * 68 + m + c);
            y0 = fmaf(v, x.x, y0); y1 = fmaf(v, x.y, y1);
        }
        *reinterpret_cast<float2*>(As + (m + r) * 68 + m + 16 + c) = make_float2(y0, y1);
        __syncthreads();
        y0 = y1 = 0.0f;
#pragma unroll
        for (int k = 0; k < 16; ++k) {
            const float v = Xs[(m + 16 + r) * 68 + m + 16 + k];
            const float2 y = *reinterpret_cast<const float2*>(As + (m + k) * 68 + m + 16 + c);
            y0 = fmaf(v, y.x, y0); y1 = fmaf(v, y.y, y1);
        }
        *reinterpret_cast<float2*>(Xs + (m + 16 + r) * 68 + m + c) = make_float2(-y0, -y1);
    }
    __syncthreads();
    {
        const int r = tid >> 3, c = (tid & 7) * 4;
        float4 y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            const float v = As[(32 + r) * 68 + k];
            const float4 x = *reinterpret_cast<const float4*>(Xs + k * 68 + c);
            y.x = fmaf(v, x.x, y.x); y.y = fmaf(v, x.y, y.y); y.z = fmaf(v, x.z, y.z); y.w = fmaf(v, x.w, y.w);
        }
        *reinterpret_cast<float4*>(As + r * 68 + 32 + c) = y;
        __syncthreads();
        y = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
        for (int k = 0; k < 32; ++k) {
            const float v = Xs[(32 + r) * 68 + 32 + k];
            const float4 x = *reinterpret_cast<const float4*>(As + k * 68 + 32 + c);
            y.x = fmaf(v, x.x, y.x); y.y = fmaf(v, x.y, y.y); y.z = fmaf(v, x.z, y.z); y.w = fmaf(v, x.w, y.w);
        }
        *reinterpret_cast<float4*>(Xs + (32 + r) * 68 + c) = make_float4(-y.x, -y.y, -y.z, -y.w);
    }
    __syncthreads();
    __nv_bfloat16* Th = reinterpret_cast<__nv_bfloat16*>(out);
    for (int i = tid; i < RC_C * 8; i += 256) {
        const int r = i >> 3, c = (i & 7) * 8;
        float v[8], lo[8];
        load_f32x8(Xs + r * 68 + c, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) lo[e] = v[e] - __bfloat162float(__float2bfloat16_rn(v[e]));
        store_f32x8(Th + r * RC_P + c, v);
        store_f32x8(Th + RC_MAT / 2 + r * RC_P + c, lo);
    }
}

// two fp32 numbers as bf16 pairs: hi + lo
__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    hi = pack_bf16x2(a, b);
    lo = pack_bf16x2(a - bf16lo(hi), b - bf16hi(hi));
}
__device__ __forceinline__ uint32_t rc_movmatrix(uint32_t x) {
    uint32_t y;
    asm volatile("movmatrix.sync.aligned.m8n8.trans.b16 %0, %1;" : "=r"(y) : "r"(x));
    return y;
}

// A CTA owns 16 or 32 columns of one head's state and walks the segment's chunks.  Every product is taken transposed - rows are
// state columns, 16 per group of four warps - so that the state, U and its right-hand side turn from accumulators into
// left operands without a change of order: they pass through shared memory as bf16 pairs (hi, lo).  The four warps of a group
// share the tokens of a chunk (16 each) for O and U and the key components (a quarter each) for the state, whose fp32 values
// stay in their registers.  K and Q (slabs of 64 components in the 128-byte swizzle), V and the chunk matrices come in two
// stages by bulk and TMA copies of a warp of its own (a copy takes its thread 140 cycles to issue), whose waits are bounded; a segment's last, short chunk and heads that do not
// fill their instance by 16-byte copies of all threads, which write zeros where there is nothing.  KT: 16-wide steps of the key components.
template <int KT, bool DELTA>
__global__ void __launch_bounds__(288) rec_chunk_kernel(const __grid_constant__ CUtensorMap map_qk, const __grid_constant__ CUtensorMap map_v, RecArgs a, RecDims d,
                                                       const int32_t* __restrict__ seg_chunk0, const uint8_t* __restrict__ ws, int* err) {
    constexpr int KP = KT * 16 + 8, PAIRS = KT >= 4 ? KT / 4 : 1;  // pairs of 8 key components of the state per warp
    constexpr int SLABS = KT >= 4 ? KT / 4 : 1, TILE = SLABS * RC_SLAB;  // K or Q of a chunk
    extern __shared__ uint8_t rc_raw[];
    uint8_t* rc_dyn = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(rc_raw) + 1023) & ~uintptr_t(1023));
    __shared__ __align__(8) uint64_t full[2];
    __shared__ int abort_flag;
    chain_trigger();
    const int tid = threadIdx.x, nthr = blockDim.x, warp = tid >> 5, lane = tid & 31, cols = (nthr - 32) / 8;
    const bool loader = tid >= nthr - 32;
    const int block = rc_block(DELTA), v_bytes = RC_C * cols * 2, stage_bytes = rc_stage(TILE, cols, DELTA);
    __nv_bfloat16* Sh = reinterpret_cast<__nv_bfloat16*>(rc_dyn + 2 * stage_bytes);  // [cols][KP]: state, hi
    __nv_bfloat16* Sl = Sh + cols * KP;
    __nv_bfloat16* Uh = Sl + cols * KP;      // [cols][RC_P]: U
    __nv_bfloat16* Wh = Uh + cols * RC_P;    // f3 U, hi and lo
    __nv_bfloat16* Wl = Wh + cols * RC_P;
    __nv_bfloat16* Rh = Wl + cols * RC_P;    // right-hand side of U, hi and lo (delta rule)
    __nv_bfloat16* Rl = Rh + cols * RC_P;
    if (tid == 0) {
        abort_flag = 0;
        tc::mbar_init(&full[0], 1);
        tc::mbar_init(&full[1], 1);
        tc::mbar_fence_init();
        tc::tma_prefetch_desc(&map_qk);
        tc::tma_prefetch_desc(&map_v);
    }
    __syncthreads();
    chain_wait();
    const int h = blockIdx.y, g = h / (d.H / d.G), seg = blockIdx.z, kp = d.kp(), vp = d.vp(), cc = d.conv_cols();
    const int c0 = blockIdx.x * cols, n_cols = min(cols, vp - c0);
    const int start = a.seg_start[seg], len = a.seg_len[seg], n_chunks = (len + RC_C - 1) / RC_C;
    const uint8_t* blocks = ws + ((long long)seg_chunk0[seg] * d.H + h) * block;
    const __nv_bfloat16* qkv = static_cast<const __nv_bfloat16*>(a.qkv) + (long long)start * cc;
    auto load = [&](int ci) {
        uint8_t* st = rc_dyn + (ci & 1) * stage_bytes;
        const int n = min(RC_C, len - ci * RC_C);
        const bool tiles = n == RC_C && kp == KT * 16;
        if (loader && lane == 0) {
            uint64_t* bar = &full[ci & 1];
            tc::mbar_expect_tx(bar, (uint32_t)(block + (tiles ? 2 * TILE + v_bytes : 0)));
            if (tiles) {
                const int y = start + ci * RC_C;
#pragma unroll
                for (int s = 0; s < SLABS; ++s) {
                    tc::tma_load_2d(st + s * RC_SLAB, &map_qk, (d.G + g) * kp + s * 64, y, bar);
                    tc::tma_load_2d(st + TILE + s * RC_SLAB, &map_qk, g * kp + s * 64, y, bar);
                }
                tc::tma_load_2d(st + 2 * TILE, &map_v, 2 * d.G * kp + h * vp + c0, y, bar);  // (columns behind the head end in state columns that do not exist)
            }
            tc::bulk_load(st + 2 * TILE + v_bytes, blocks + (long long)ci * d.H * block, block, bar);
        }
        if (!tiles) {
            const __nv_bfloat16* rows = qkv + (long long)ci * RC_C * cc;
            for (int i = tid; i < 2 * RC_C * KT * 2; i += nthr) {  // k, then q
                const int q = i / (RC_C * KT * 2), r = i / (KT * 2) % RC_C, c = i % (KT * 2) * 8;
                const bool on = r < n && c < kp;
                cp_async16(smem_u32(st + q * TILE + (c >> 6) * RC_SLAB + r * 128 + ((((c >> 3) & 7) ^ (r & 7)) << 4)),
                           on ? rows + (long long)r * cc + ((q ? 0 : d.G) + g) * kp + c : rows, on);
            }
            for (int i = tid; i < RC_C * (cols / 8); i += nthr) {
                const int r = i / (cols / 8), c = i % (cols / 8) * 8;
                const bool on = r < n && c < n_cols;
                cp_async16(smem_u32(st + 2 * TILE + (r * cols + c) * 2), on ? rows + (long long)r * cc + 2 * d.G * kp + h * vp + c0 + c : rows, on);
            }
        }
        cp_async_commit();
    };
    load(0);
    const int mt = warp >> 2, w = warp & 3;
    const int jp = mt & 1 ? 3 - w : w;  // this warp's tokens of a chunk: 16 jp .. 16 jp + 15 (the triangles even out over the schedulers)
    const int lm = lane >> 3, lr = lane & 7, kc = (lane & 3) * 2, ar = mt * 16 + (lane >> 2);
    // accumulators: row (lane / 4, + 8) = state column, columns (lane % 4) * 2, + 1 = token or key component
    float* state = a.S + ((long long)a.seg_slot[seg] * d.H + h) * kp * vp;
    const bool fresh = a.seg_pos0[seg] == 0, keeps = !loader && w * PAIRS < KT;
    float S[2 * PAIRS][4];
#pragma unroll
    for (int j = 0; j < 2 * PAIRS; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int k = (w * 2 * PAIRS + j) * 8 + kc + (e & 1), c = c0 + ar + (e >> 1) * 8;
            S[j][e] = keeps && !fresh && k < kp && c < vp ? state[(long long)k * vp + c] : 0.0f;
        }
    auto publish = [&](__nv_bfloat16* hi, __nv_bfloat16* lo, int pitch, int col, const float (&v)[4]) {
        uint32_t h0, l0, h1, l1;
        split2(v[0], v[1], h0, l0);
        split2(v[2], v[3], h1, l1);
        *reinterpret_cast<uint32_t*>(hi + ar * pitch + col + kc) = h0;
        *reinterpret_cast<uint32_t*>(hi + (ar + 8) * pitch + col + kc) = h1;
        *reinterpret_cast<uint32_t*>(lo + ar * pitch + col + kc) = l0;
        *reinterpret_cast<uint32_t*>(lo + (ar + 8) * pitch + col + kc) = l1;
    };
    auto publish_state = [&]() {
        if (keeps)
#pragma unroll
            for (int j = 0; j < 2 * PAIRS; ++j) publish(Sh, Sl, KP, (w * 2 * PAIRS + j) * 8, S[j]);
    };
    publish_state();
    const int a_row = mt * 16 + (lm & 1) * 8 + lr, a_col = (lm >> 1) * 8;   // left operand: matrices = rows 0-7 / 8-15 (lm & 1), columns + 8 (lm >> 1)
    const int b_row = (lm >> 1) * 8 + lr, b_col = (lm & 1) * 8;             // right operand, row = output column
    const uint32_t sh = smem_u32(Sh + a_row * KP + a_col), sl = smem_u32(Sl + a_row * KP + a_col);
    const uint32_t uh = smem_u32(Uh + a_row * RC_P + a_col), wh = smem_u32(Wh + a_row * RC_P + a_col), wl = smem_u32(Wl + a_row * RC_P + a_col);
    const uint32_t rh = smem_u32(Rh + a_row * RC_P + a_col), rl = smem_u32(Rl + a_row * RC_P + a_col);
    bool ok = true;
    for (int ci = 0; ci < n_chunks; ++ci) {
        cp_async_wait<0>();
        __syncthreads();  // K, Q, V are here, the state is published, the other stage used up
        if (ci + 1 < n_chunks) load(ci + 1);
        if (loader) {
            if (DELTA && !__syncthreads_and(1)) { ok = false; break; }
            if (!__syncthreads_and(1)) { ok = false; break; }
            continue;
        }
        ok = tc::mbar_wait(&full[ci & 1], (ci >> 1) & 1, &abort_flag, err, RC_ERR_FULL);
        const uint8_t* st = rc_dyn + (ci & 1) * stage_bytes;
        const uint32_t kb = smem_u32(st), qb = kb + TILE, vb = qb + TILE, tb = vb + v_bytes;
        const uint32_t pm = tb + (DELTA ? 2 * RC_MAT : 0) + ((jp * 16 + b_row) * RC_P + b_col) * 2;
        const float* f = reinterpret_cast<const float*>(st + 2 * TILE + v_bytes + (DELTA ? 3 : 1) * RC_MAT);
        float u[2][4], o[2][4];
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            u[x][0] = u[x][1] = u[x][2] = u[x][3] = 0.0f;
            o[x][0] = o[x][1] = o[x][2] = o[x][3] = 0.0f;
        }
        // S0^T K^T and S0^T Q^T of this warp's tokens
        const uint32_t k_addr = kb + (jp * 16 + b_row) * 128, q_addr = qb + (jp * 16 + b_row) * 128, x0 = (lm & 1) ^ lr;  // (the row's piece p lies at p ^ lr)
#pragma unroll
        for (int kk = 0; kk < KT; ++kk) {
            uint32_t hi[4], lo[4], b[4];
            ldsm_x4(sh + kk * 32, hi);
            ldsm_x4(sl + kk * 32, lo);
            const uint32_t piece = (kk >> 2) * RC_SLAB + ((((kk & 3) * 2) ^ x0) << 4);
            ldsm_x4(q_addr + piece, b);
            mma_16816(o[0], hi, b[0], b[1]);
            mma_16816(o[1], hi, b[2], b[3]);
            mma_16816(o[0], lo, b[0], b[1]);
            mma_16816(o[1], lo, b[2], b[3]);
            if (DELTA) {
                ldsm_x4(k_addr + piece, b);
                mma_16816(u[0], hi, b[0], b[1]);
                mma_16816(u[1], hi, b[2], b[3]);
                mma_16816(u[0], lo, b[0], b[1]);
                mma_16816(u[1], lo, b[2], b[3]);
            }
        }
        {   // right-hand side: f0 v - f1 (K S0); the decayed sum has U = v
            uint32_t v[4];  // matrices: tokens 0-7 / 8-15 (lm >> 1), state columns + 8 (lm & 1); transposed
            ldsm_x4_trans(vb + (jp * 16 + b_row) * cols * 2 + mt * 32 + b_col * 2, v);
#pragma unroll
            for (int x = 0; x < 2; ++x) {
                const int t = jp * 16 + x * 8;
                float2 fk = make_float2(0.0f, 0.0f);
                const float2 fv = *reinterpret_cast<const float2*>(f + t + kc);
                if (DELTA) fk = *reinterpret_cast<const float2*>(f + RC_C + t + kc);
                u[x][0] = fv.x * bf16lo(v[2 * x]) - fk.x * u[x][0];
                u[x][1] = fv.y * bf16hi(v[2 * x]) - fk.y * u[x][1];
                u[x][2] = fv.x * bf16lo(v[2 * x + 1]) - fk.x * u[x][2];
                u[x][3] = fv.y * bf16hi(v[2 * x + 1]) - fk.y * u[x][3];
                if (DELTA) publish(Rh, Rl, RC_P, t, u[x]);
            }
        }
        if (DELTA) {  // U = T R
            if (!__syncthreads_and(ok)) { ok = false; break; }
            const uint32_t t_addr = tb + ((jp * 16 + b_row) * RC_P + b_col) * 2;
#pragma unroll
            for (int x = 0; x < 2; ++x) u[x][0] = u[x][1] = u[x][2] = u[x][3] = 0.0f;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                if (kk > jp) break;  // (lower triangle)
                uint32_t hi[4], lo[4], b[4], c[4];
                ldsm_x4(rh + kk * 32, hi);
                ldsm_x4(rl + kk * 32, lo);
                ldsm_x4(t_addr + kk * 32, b);
                ldsm_x4(t_addr + RC_MAT + kk * 32, c);
                mma_16816(u[0], hi, b[0], b[1]);
                mma_16816(u[1], hi, b[2], b[3]);
                mma_16816(u[0], lo, b[0], b[1]);
                mma_16816(u[1], lo, b[2], b[3]);
                mma_16816(u[0], hi, c[0], c[1]);
                mma_16816(u[1], hi, c[2], c[3]);
            }
        }
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const int t = jp * 16 + x * 8;
            const float2 fs = *reinterpret_cast<const float2*>(f + 3 * RC_C + t + kc);
            *reinterpret_cast<uint32_t*>(Uh + ar * RC_P + t + kc) = pack_bf16x2(u[x][0], u[x][1]);
            *reinterpret_cast<uint32_t*>(Uh + (ar + 8) * RC_P + t + kc) = pack_bf16x2(u[x][2], u[x][3]);
            const float scaled[4] = {u[x][0] * fs.x, u[x][1] * fs.y, u[x][2] * fs.x, u[x][3] * fs.y};
            publish(Wh, Wl, RC_P, t, scaled);
        }
        if (!__syncthreads_and(ok)) { ok = false; break; }
        // S = decay S0 + (f3 U)^T K, this warp's key components
        if (keeps) {
            const float decay = f[4 * RC_C];
#pragma unroll
            for (int j = 0; j < 2 * PAIRS; ++j)
#pragma unroll
                for (int e = 0; e < 4; ++e) S[j][e] *= decay;
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                uint32_t hi[4], lo[4];
                ldsm_x4(wh + kk * 32, hi);
                ldsm_x4(wl + kk * 32, lo);
#pragma unroll
                for (int i = 0; i < PAIRS; ++i) {
                    uint32_t b[4];  // matrices: tokens 0-7 / 8-15 (lm & 1), components + 8 (lm >> 1); transposed
                    const int pair = w * PAIRS + i;
                    ldsm_x4_trans(kb + (pair >> 2) * RC_SLAB + (kk * 16 + (lm & 1) * 8 + lr) * 128 + ((((pair & 3) * 2) ^ (lm >> 1) ^ lr) << 4), b);
                    mma_16816(S[2 * i], hi, b[0], b[1]);
                    mma_16816(S[2 * i + 1], hi, b[2], b[3]);
                    mma_16816(S[2 * i], lo, b[0], b[1]);
                    mma_16816(S[2 * i + 1], lo, b[2], b[3]);
                }
            }
            publish_state();
        }
        // O = f2 (Q S0) + P U
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const float2 fq = *reinterpret_cast<const float2*>(f + 2 * RC_C + jp * 16 + x * 8 + kc);
            o[x][0] *= fq.x; o[x][1] *= fq.y; o[x][2] *= fq.x; o[x][3] *= fq.y;
        }
#pragma unroll
        for (int kk = 0; kk < 4; ++kk) {
            if (kk > jp) break;
            uint32_t hi[4], b[4];
            ldsm_x4(uh + kk * 32, hi);
            ldsm_x4(pm + kk * 32, b);
            mma_16816(o[0], hi, b[0], b[1]);
            mma_16816(o[1], hi, b[2], b[3]);
        }
        // output rows: tokens, this group's columns
        const int n = len - ci * RC_C, col = c0 + mt * 16 + kc;
        __nv_bfloat16* out = static_cast<__nv_bfloat16*>(a.out) + (long long)(start + ci * RC_C) * d.H * vp + h * vp + col;
#pragma unroll
        for (int x = 0; x < 2; ++x) {
            const uint32_t w0 = rc_movmatrix(pack_bf16x2(o[x][0], o[x][1])), w1 = rc_movmatrix(pack_bf16x2(o[x][2], o[x][3]));
            const int t = jp * 16 + x * 8 + (lane >> 2);
            if (t < n) {
                if (col < vp) *reinterpret_cast<uint32_t*>(out + (long long)t * d.H * vp) = w0;
                if (col + 8 < vp) *reinterpret_cast<uint32_t*>(out + (long long)t * d.H * vp + 8) = w1;
            }
        }
    }
    if (!ok) {  // a copy did not arrive: let the ones in flight land (bounded); the host learns of it
        if (tid == 0) {
            const long long t = clock64();
            while (clock64() - t < tc::WAIT_LIMIT_CYCLES / 4) {}
        }
        __syncthreads();
        return;
    }
    if (keeps)
#pragma unroll
        for (int j = 0; j < 2 * PAIRS; ++j)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int k = (w * 2 * PAIRS + j) * 8 + kc + (e & 1), c = c0 + ar + (e >> 1) * 8;
                if (k < kp && c < vp) state[(long long)k * vp + c] = S[j][e];
            }
}

// ---- decode step: one token per segment ---------------------------------------------------------------------------
// A CTA per (head, sequence).  The state passes through shared memory, in and out by one bulk copy each (IN_SMEM; larger states
// are read twice from global memory); it is requested before the predecessor kernel ends - only this kernel writes it, and
// passes are separated by the host.  Both products S^T k and S^T q come from one pass over the old state:
//     S^T k of the decayed state = g (S^T k),   o = g (S^T q) + (k . q) u.
// The delta rule's CTA has the whole head: it also takes beta and the decay from the layer's input x (two dot products) and
// applies the norm and the gate, so that its output is the operand of the output projection.
constexpr int RT_THREADS = 256;
constexpr int RT_ERR_FULL = 72;
constexpr int RT_MAX_SMEM = 200 * 1024;

template <typename T, bool IN_SMEM, bool DELTA>
__global__ void __launch_bounds__(RT_THREADS, 3) rec_step_kernel(RecArgs a, RecDims d, int lpr, int* err) {
    extern __shared__ __align__(16) float rt_sm[];  // [state [kp][vp] |] partial sums [2][row groups][vp], q [kp], k [kp], o [vp]
    __shared__ float red[RT_THREADS / 32][5], tot[5];
    __shared__ __align__(8) uint64_t full;
    __shared__ int abort_flag;
    const int kp = d.kp(), vp = d.vp(), groups = RT_THREADS / lpr;
    float *pk = rt_sm + (IN_SMEM ? kp * vp : 0), *pq = pk + groups * vp, *qs = pq + groups * vp, *ks = qs + kp, *os = ks + kp;
    chain_trigger();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x, g = h / (d.H / d.G), seg = blockIdx.y;
    const int rg = tid / lpr, c = (tid % lpr) * 4;
    const bool on = c < vp;
    const bool fresh = a.seg_pos0[seg] == 0;
    float* state = a.S + ((long long)a.seg_slot[seg] * d.H + h) * kp * vp;
    if (IN_SMEM) {
        if (fresh) {
            for (int i = tid; i < kp * vp / 4; i += RT_THREADS) reinterpret_cast<float4*>(rt_sm)[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        } else if (tid == 0) {
            abort_flag = 0;
            tc::mbar_init(&full, 1);
            tc::mbar_fence_init();
            tc::mbar_expect_tx(&full, (uint32_t)(kp * vp * 4));
            tc::bulk_load(rt_sm, state, (uint32_t)(kp * vp * 4), &full);
        }
    }
    const float A = DELTA ? a.A[h] : a.decay[h], dt_bias = DELTA ? a.dt_bias[h] : 0.0f;
    const float gain = DELTA && tid < vp ? a.norm[tid] : 0.0f;
    chain_wait();
    const int t = seg;  // every segment is one token
    const T* row = static_cast<const T*>(a.qkv) + (long long)t * d.conv_cols();
    const T* z = static_cast<const T*>(a.z) + (long long)t * d.raw_cols() + h * vp;
    // this thread's first column of v and z: requested here, used much later
    const float v0 = tid < vp ? to_f32(row[2 * d.G * kp + h * vp + tid]) : 0.0f, z0 = DELTA && tid < vp ? to_f32(z[tid]) : 0.0f;
    float sums[5] = {0.f, 0.f, 0.f, 0.f, 0.f};  // q . q, k . k, q . k, b, a
    for (int i = tid; i < kp; i += RT_THREADS) {
        const float q = to_f32(row[g * kp + i]), k = to_f32(row[(d.G + g) * kp + i]);
        qs[i] = q; ks[i] = k;
        sums[0] = fmaf(q, q, sums[0]); sums[1] = fmaf(k, k, sums[1]); sums[2] = fmaf(q, k, sums[2]);
    }
    if (DELTA) {
        const T* x = static_cast<const T*>(a.x) + (long long)t * a.x_pitch;
        const T* wb = static_cast<const T*>(a.ba_w) + (long long)h * a.x_pitch;
        const T* wa = wb + (long long)(d.ba_cols() / 2) * a.x_pitch;
#pragma unroll 2
        for (int i = tid * 8; i < a.x_pitch; i += RT_THREADS * 8) {
            float xv[8], bv[8], av[8];
            load_f32x8(x + i, xv); load_f32x8(wb + i, bv); load_f32x8(wa + i, av);
#pragma unroll
            for (int e = 0; e < 8; ++e) { sums[3] = fmaf(xv[e], bv[e], sums[3]); sums[4] = fmaf(xv[e], av[e], sums[4]); }
        }
    }
#pragma unroll
    for (int i = 0; i < (DELTA ? 5 : 3); ++i) {
        sums[i] = warp_sum(sums[i]);
        if (lane == 0) red[warp][i] = sums[i];
    }
    __syncthreads();
    if (tid < (DELTA ? 5 : 3)) {
        float s = 0.0f;
#pragma unroll
        for (int w = 0; w < RT_THREADS / 32; ++w) s += red[w][tid];
        tot[tid] = s;
    }
    if (IN_SMEM && !fresh && !__syncthreads_and(tc::mbar_wait(&full, 0, &abort_flag, err, RT_ERR_FULL))) {
        if (tid == 0) {  // let the copy in flight land (bounded); the host learns of it
            const long long t0 = clock64();
            while (!tc::mbar_try_wait(&full, 0) && clock64() - t0 < tc::WAIT_LIMIT_CYCLES) {}
        }
        __syncthreads();
        return;
    }
    const float* old = IN_SMEM ? rt_sm : state;
    if (on) {
        float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
        if (IN_SMEM || !fresh)
#pragma unroll 4
            for (int r = rg; r < kp; r += groups) {
                const float4 s = *reinterpret_cast<const float4*>(old + r * vp + c);
                const float k = ks[r], q = qs[r];
                ak.x = fmaf(s.x, k, ak.x); ak.y = fmaf(s.y, k, ak.y); ak.z = fmaf(s.z, k, ak.z); ak.w = fmaf(s.w, k, ak.w);
                aq.x = fmaf(s.x, q, aq.x); aq.y = fmaf(s.y, q, aq.y); aq.z = fmaf(s.z, q, aq.z); aq.w = fmaf(s.w, q, aq.w);
            }
        *reinterpret_cast<float4*>(pk + rg * vp + c) = ak;
        *reinterpret_cast<float4*>(pq + rg * vp + c) = aq;
    }
    __syncthreads();
    const float nq = DELTA ? a.q_scale / sqrtf(tot[0] + UNIT_EPS) : 1.0f, nk = DELTA ? 1.0f / sqrtf(tot[1] + UNIT_EPS) : 1.0f;
    const float beta = DELTA ? rec_sigmoid(tot[3]) : 1.0f;
    const float gt = DELTA ? expf(A * rec_softplus(tot[4] + dt_bias)) : A;
    const float kq = tot[2] * nk * nq;
    // one thread per column: fold the row groups, the new value u and the output
    float ss = 0.0f;
    for (int j = tid; j < vp; j += RT_THREADS) {
        float sk = 0.0f, sq = 0.0f;
        for (int r = 0; r < groups; ++r) { sk += pk[r * vp + j]; sq += pq[r * vp + j]; }
        float u = j == tid ? v0 : to_f32(row[2 * d.G * kp + h * vp + j]);
        if (DELTA) u = beta * (u - gt * nk * sk);
        const float o = fmaf(kq, u, gt * nq * sq);
        os[j] = o;
        ss = fmaf(o, o, ss);
        pk[j] = u * nk;  // (row group 0 of this column has been read)
    }
    if (DELTA) {
        ss = warp_sum(ss);
        if (lane == 0) red[warp][0] = ss;
    }
    __syncthreads();
    if (on) {
        const float4 u = *reinterpret_cast<const float4*>(pk + c);
#pragma unroll 4
        for (int r = rg; r < kp; r += groups) {
            float4 s = IN_SMEM || !fresh ? *reinterpret_cast<const float4*>(old + r * vp + c) : make_float4(0.f, 0.f, 0.f, 0.f);
            const float k = ks[r];
            s.x = fmaf(k, u.x, gt * s.x); s.y = fmaf(k, u.y, gt * s.y); s.z = fmaf(k, u.z, gt * s.z); s.w = fmaf(k, u.w, gt * s.w);
            *reinterpret_cast<float4*>((IN_SMEM ? rt_sm : state) + r * vp + c) = s;
        }
    }
    if (IN_SMEM) {
        tc::fence_proxy_async_smem();
        __syncthreads();
        if (tid == 0) {
            asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(reinterpret_cast<uint64_t>(state)), "r"(smem_u32(rt_sm)), "r"(kp * vp * 4)
                         : "memory");
            asm volatile("cp.async.bulk.commit_group;" ::: "memory");
        }
    }
    T* out = static_cast<T*>(a.out) + (long long)t * d.H * vp + h * vp;
    if (DELTA) {
        ss = 0.0f;
#pragma unroll
        for (int w = 0; w < RT_THREADS / 32; ++w) ss += red[w][0];
    }
    const float rms = DELTA ? sqrtf(ss / (float)d.dv + a.eps) : 1.0f;
    for (int j = tid; j < vp; j += RT_THREADS) {
        float o = os[j];
        if (DELTA) {
            const float zv = j == tid ? z0 : to_f32(z[j]);
            o = o / rms * (j == tid ? gain : a.norm[j]) * (zv * rec_sigmoid(zv));
        }
        out[j] = from_f32<T>(o);
    }
    if (IN_SMEM && tid == 0) asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");  // the copy out reads this CTA's memory
}

// ---- norm and gate of the output ----------------------------------------------------------------------------------
// PER_HEAD: every head by itself, weight [vp], gate silu(z); otherwise all heads together, weight [H vp], gate sigmoid(z).
// In place.  One CTA per token; a thread holds MAXV vectors of eight columns (0: any number, read twice).  PER_HEAD with MAXV > 0
// needs heads of 8 x 2^n <= 256 columns: a head is a group of neighbouring lanes.
template <typename T>
__device__ __forceinline__ float gate_sigmoid(float x) {
    if constexpr (sizeof(T) == 4) return rec_sigmoid(x);
    return fast_rcp(1.0f + fast_ex2(-LOG2E * x));
}
template <typename T, bool PER_HEAD, int MAXV>
__global__ void __launch_bounds__(256) rec_norm_kernel(T* __restrict__ o, const T* __restrict__ z, long long z_pitch, const float* __restrict__ gain,
                                                       float eps, int H, int dv, int vp) {
    __shared__ float red[8];
    chain_trigger();
    chain_wait();
    T* row = o + (long long)blockIdx.x * H * vp;
    const T* zr = z + blockIdx.x * z_pitch;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, n = H * vp;
    if constexpr (PER_HEAD && MAXV == 0) {
        for (int h = warp; h < H; h += 8) {
            float ss = 0.0f;
            for (int j = lane * 2; j < vp; j += 64) {
                float a, b;
                load_f32x2(row + h * vp + j, a, b);
                ss = fmaf(a, a, fmaf(b, b, ss));
            }
            const float rms = sqrtf(warp_sum(ss) / (float)dv + eps);
            for (int j = lane * 2; j < vp; j += 64) {
                float a, b, za, zb;
                load_f32x2(row + h * vp + j, a, b);
                load_f32x2(zr + h * vp + j, za, zb);
                store_f32x2(row + h * vp + j, a / rms * gain[j] * (za * gate_sigmoid<T>(za)), b / rms * gain[j + 1] * (zb * gate_sigmoid<T>(zb)));
            }
        }
        return;
    } else {
        float v[MAXV ? MAXV : 1][8], zv[MAXV ? MAXV : 1][8], ss[MAXV ? MAXV : 1], all = 0.0f;
        if constexpr (MAXV > 0) {
#pragma unroll
            for (int i = 0; i < MAXV; ++i) {
                const int j = (i * 256 + threadIdx.x) * 8;
                ss[i] = 0.0f;
                if (j < n) {
                    load_f32x8(row + j, v[i]);
                    load_f32x8(zr + j, zv[i]);
#pragma unroll
                    for (int e = 0; e < 8; ++e) ss[i] = fmaf(v[i][e], v[i][e], ss[i]);
                }
                all += ss[i];
            }
        } else {
            for (int j = threadIdx.x * 8; j < n; j += 2048) {
                load_f32x8(row + j, v[0]);
#pragma unroll
                for (int e = 0; e < 8; ++e) all = fmaf(v[0][e], v[0][e], all);
            }
        }
        if (!PER_HEAD) {
            all = warp_sum(all);
            if (lane == 0) red[warp] = all;
            __syncthreads();
            all = 0.0f;
#pragma unroll
            for (int w = 0; w < 8; ++w) all += red[w];
        }
        auto finish = [&](int j, float (&x)[8], const float (&zz)[8], float sum) {
            const float inv = 1.0f / sqrtf(sum / (float)(PER_HEAD ? dv : H * dv) + eps);
            float gv[8];
            load_f32x8(gain + (PER_HEAD ? j % vp : j), gv);
#pragma unroll
            for (int e = 0; e < 8; ++e) x[e] = x[e] * inv * gv[e] * (PER_HEAD ? zz[e] * gate_sigmoid<T>(zz[e]) : gate_sigmoid<T>(zz[e]));
            store_f32x8(row + j, x);
        };
        if constexpr (MAXV > 0) {
#pragma unroll
            for (int i = 0; i < MAXV; ++i) {
                const int j = (i * 256 + threadIdx.x) * 8;
                if (PER_HEAD)
                    for (int x = 1; x < vp / 8; x <<= 1) ss[i] += __shfl_xor_sync(0xffffffffu, ss[i], x);
                if (j < n) finish(j, v[i], zv[i], PER_HEAD ? ss[i] : all);
            }
        } else {
            for (int j = threadIdx.x * 8; j < n; j += 2048) {
                load_f32x8(row + j, v[0]);
                load_f32x8(zr + j, zv[0]);
                finish(j, v[0], zv[0], all);
            }
        }
    }
}

// ---- launches -----------------------------------------------------------------------------------------------------
static RecArgs rec_args(bool f32, const RecDims& d, const RecWeights& w, const RecState& s, const StepTokens& tk, const void* raw, const void* qkv, void* out,
                        float eps) {
    RecArgs a{};
    a.qkv = qkv;
    a.z = static_cast<const char*>(raw) + (size_t)d.conv_cols() * (f32 ? 4 : 2);
    a.A = w.A; a.dt_bias = w.dt_bias; a.decay = w.decay; a.log_decay = w.log_decay; a.norm = w.norm; a.ba_w = w.ba;
    a.S = s.S; a.out = out;
    a.seg_start = tk.seg_start; a.seg_len = tk.seg_len; a.seg_pos0 = tk.seg_pos0; a.seg_slot = tk.seg_slot;
    a.eps = eps; a.q_scale = 1.0f / sqrtf((float)d.dk);
    return a;
}

template <typename T, int NS, bool DELTA>
static jsm_status scan_go(const RecArgs& a, const RecDims& d, int n_segs, cudaStream_t st) {
    JSM_CUDA_CHECK(launch_chained(rec_scan_kernel<T, NS, DELTA>, dim3((d.vp() + RS_COLS - 1) / RS_COLS, d.H, n_segs), dim3(RS_THREADS), 0, st, a, d));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
template <typename T, bool DELTA>
static jsm_status scan_sized(const RecArgs& a, const RecDims& d, int n_segs, cudaStream_t st) {
    const int kp = d.kp();
    return kp <= 32 ? scan_go<T, 4, DELTA>(a, d, n_segs, st) : kp <= 64 ? scan_go<T, 8, DELTA>(a, d, n_segs, st)
         : kp <= 128 ? scan_go<T, 16, DELTA>(a, d, n_segs, st) : scan_go<T, 32, DELTA>(a, d, n_segs, st);
}

template <typename T>
static jsm_status norm_typed(const RecDims& d, const RecArgs& a, int n_tok, cudaStream_t st) {
    auto go = [&](auto kernel) {
        return launch_chained(kernel, dim3(n_tok), dim3(256), 0, st, (T*)a.out, (const T*)a.z, (long long)d.raw_cols(), a.norm, a.eps, d.H, d.dv, d.vp());
    };
    const int n = d.H * d.vp(), lanes = d.vp() / 8;
    const bool groups = lanes <= 32 && (lanes & (lanes - 1)) == 0;
    if (d.delta) JSM_CUDA_CHECK(n <= 2048 && groups ? go(rec_norm_kernel<T, true, 1>) : n <= 4096 && groups ? go(rec_norm_kernel<T, true, 2>)
                                : n <= 8192 && groups ? go(rec_norm_kernel<T, true, 4>) : go(rec_norm_kernel<T, true, 0>));
    else JSM_CUDA_CHECK(n <= 2048 ? go(rec_norm_kernel<T, false, 1>) : n <= 4096 ? go(rec_norm_kernel<T, false, 2>)
                        : n <= 8192 ? go(rec_norm_kernel<T, false, 4>) : go(rec_norm_kernel<T, false, 0>));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

bool rec_usable(const RecDims& d) { return d.dk <= 256 && d.dv <= 1024; }

// the chunk kernels: key components in 16-wide steps, rounded up to an instance
static int chunk_kt(const RecDims& d) { return d.kp() <= 32 ? 2 : d.kp() <= 64 ? 4 : 8; }
bool rec_chunk_usable(const RecDims& d) { return d.dk <= 128 && d.dv <= 1024; }
size_t rec_chunk_bytes(const RecDims& d) { return (size_t)d.H * rc_block(d.delta); }

template <int KT, bool DELTA>
static jsm_status chunk_go(const RecArgs& a, const RecDims& d, const RecChunks& ch, int n_segs, int n_tok, cudaStream_t st) {
    static bool attr_done = false;
    if (!attr_done) {
        JSM_CUDA_CHECK(cudaFuncSetAttribute(rec_chunk_prep_kernel<DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, 80 * 1024));
        JSM_CUDA_CHECK(cudaFuncSetAttribute(rec_chunk_kernel<KT, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        attr_done = true;
    }
    const int kw = KT * 16;
    JSM_CUDA_CHECK(launch_chained(rec_chunk_prep_kernel<DELTA>, dim3(ch.n_chunks, d.H), dim3(256), (size_t)rc_prep_tiles(kw, DELTA) + (DELTA ? RC_C * 68 * 4 : 0), st, a, d,
                                  ch.chunk_seg, ch.chunk_t0, static_cast<uint8_t*>(ch.ws), kw));
    JSM_LAUNCH_CHECK();
    // columns per CTA: 16 while that leaves SMs idle
    const int cols = (long long)n_segs * d.H * ((d.vp() + 15) / 16) <= sm_count() || d.vp() <= 16 ? 16 : 32;
    const size_t smem = 2 * (size_t)rc_stage((KT >= 4 ? KT / 4 : 1) * RC_SLAB, cols, DELTA) + (size_t)cols * (2 * (kw + 8) + (DELTA ? 5 : 3) * RC_P) * 2 + 1024;
    CUtensorMap map_qk, map_v;
    jsm_status s = make_tmap_bf16_2d(&map_qk, a.qkv, (uint64_t)n_tok, (uint64_t)d.conv_cols(), (uint64_t)d.conv_cols(), RC_C, 64);
    if (s != JSM_OK) return s;
    s = make_tmap_bf16_2d(&map_v, a.qkv, (uint64_t)n_tok, (uint64_t)d.conv_cols(), (uint64_t)d.conv_cols(), RC_C, cols, false);
    if (s != JSM_OK) return s;
    JSM_CUDA_CHECK(launch_chained(rec_chunk_kernel<KT, DELTA>, dim3((d.vp() + cols - 1) / cols, d.H, n_segs), dim3(cols * 8 + 32), smem, st, map_qk, map_v, a, d, ch.seg_chunk0,
                                  static_cast<const uint8_t*>(ch.ws), tc_error_word()));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
template <bool DELTA>
static jsm_status chunk_sized(const RecArgs& a, const RecDims& d, const RecChunks& ch, int n_segs, int n_tok, cudaStream_t st) {
    switch (chunk_kt(d)) {
        case 2: return chunk_go<2, DELTA>(a, d, ch, n_segs, n_tok, st);
        case 4: return chunk_go<4, DELTA>(a, d, ch, n_segs, n_tok, st);
        default: return chunk_go<8, DELTA>(a, d, ch, n_segs, n_tok, st);
    }
}

jsm_status rec_scan_launch(bool f32, const RecDims& d, const RecWeights& w, const RecState& s, float eps, const StepTokens& tk, const RecChunks& ch,
                           const void* raw, const void* qkv, const float* ba, void* out, cudaStream_t st) {
    if (!rec_usable(d)) JSM_FAIL(JSM_UNSUPPORTED, "linear recurrence: heads of %d / %d components (at most 256 / 1024)", d.dk, d.dv);
    RecArgs a = rec_args(f32, d, w, s, tk, raw, qkv, out, eps);
    a.ba = ba;
    jsm_status r;
    if (!f32 && rec_chunk_usable(d)) r = d.delta ? chunk_sized<true>(a, d, ch, tk.n_segs, tk.T, st) : chunk_sized<false>(a, d, ch, tk.n_segs, tk.T, st);
    else r = f32 ? (d.delta ? scan_sized<float, true>(a, d, tk.n_segs, st) : scan_sized<float, false>(a, d, tk.n_segs, st))
                       : (d.delta ? scan_sized<__nv_bfloat16, true>(a, d, tk.n_segs, st) : scan_sized<__nv_bfloat16, false>(a, d, tk.n_segs, st));
    if (r != JSM_OK) return r;
    return f32 ? norm_typed<float>(d, a, tk.T, st) : norm_typed<__nv_bfloat16>(d, a, tk.T, st);
}

template <typename T, bool IN_SMEM, bool DELTA>
static jsm_status step_go(const RecArgs& a, const RecDims& d, int lpr, size_t smem, int n_segs, cudaStream_t st) {
    static bool attr_done = false;
    if (!attr_done) {
        JSM_CUDA_CHECK(cudaFuncSetAttribute(rec_step_kernel<T, IN_SMEM, DELTA>, cudaFuncAttributeMaxDynamicSharedMemorySize, RT_MAX_SMEM));
        attr_done = true;
    }
    JSM_CUDA_CHECK(launch_chained(rec_step_kernel<T, IN_SMEM, DELTA>, dim3(d.H, n_segs), dim3(RT_THREADS), smem, st, a, d, lpr, tc_error_word()));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
template <typename T, bool DELTA>
static jsm_status step_sized(const RecArgs& a, const RecDims& d, int n_segs, cudaStream_t st) {
    int lpr = 1;  // lanes per row of the state
    while (lpr * 4 < d.vp()) lpr *= 2;
    const size_t base = sizeof(float) * (2 * d.kp() + 2 * (size_t)(RT_THREADS / lpr) * d.vp() + d.vp()), state = sizeof(float) * d.kp() * d.vp();
    return base + state <= RT_MAX_SMEM ? step_go<T, true, DELTA>(a, d, lpr, base + state, n_segs, st) : step_go<T, false, DELTA>(a, d, lpr, base, n_segs, st);
}

jsm_status rec_step_launch(bool f32, const RecDims& d, const RecWeights& w, const RecState& s, float eps, const StepTokens& tk, const void* raw,
                           const void* qkv, const void* x, int x_pitch, void* out, cudaStream_t st) {
    if (!rec_usable(d)) JSM_FAIL(JSM_UNSUPPORTED, "linear recurrence: heads of %d / %d components (at most 256 / 1024)", d.dk, d.dv);
    RecArgs a = rec_args(f32, d, w, s, tk, raw, qkv, out, eps);
    a.x = x; a.x_pitch = x_pitch;
    jsm_status r = f32 ? (d.delta ? step_sized<float, true>(a, d, tk.n_segs, st) : step_sized<float, false>(a, d, tk.n_segs, st))
                       : (d.delta ? step_sized<__nv_bfloat16, true>(a, d, tk.n_segs, st) : step_sized<__nv_bfloat16, false>(a, d, tk.n_segs, st));
    if (r != JSM_OK || d.delta) return r;
    return f32 ? norm_typed<float>(d, a, tk.T, st) : norm_typed<__nv_bfloat16>(d, a, tk.T, st);
}

}  // namespace jsm
