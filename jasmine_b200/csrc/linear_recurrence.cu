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
// Row of the input projection: [q: G heads | k: G heads | v: H heads | z: H heads], heads at pitches padded to 8; head h uses
// query / key head h / (H / G).  State: [slot][head][kp][vp].
#include "decoder_ops.cuh"
#include "mma_utils.cuh"
#include <math.h>
#include <algorithm>

namespace jsm {

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

// ---- decode step: one token per segment ---------------------------------------------------------------------------
// A CTA per (head, sequence).  A thread owns four columns of NR rows of the state (0: any number, read twice); the state is
// requested before the predecessor kernel ends - only this kernel writes it, and passes are separated by the host.  Both
// products S^T k and S^T q come from one pass over the old state:
//     S^T k of the decayed state = g (S^T k),   o = g (S^T q) + (k . q) u.
// The delta rule's CTA has the whole head: it also takes beta and the decay from the layer's input x (two dot products) and
// applies the norm and the gate, so that its output is the operand of the output projection.
constexpr int RT_THREADS = 256;

template <typename T, int NR, bool DELTA>
__global__ void __launch_bounds__(RT_THREADS) rec_step_kernel(RecArgs a, RecDims d, int lpr) {
    extern __shared__ float rt_sm[];  // q [kp], k [kp], partial sums [2][row groups][vp], o [vp]
    __shared__ float red[RT_THREADS / 32][5], tot[5];
    const int kp = d.kp(), vp = d.vp(), groups = RT_THREADS / lpr;
    float *qs = rt_sm, *ks = qs + kp, *pk = ks + kp, *pq = pk + groups * vp, *os = pq + groups * vp;
    chain_trigger();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.x, g = h / (d.H / d.G), seg = blockIdx.y;
    const int rg = tid / lpr, c = (tid % lpr) * 4;
    const bool on = c < vp;
    const bool fresh = a.seg_pos0[seg] == 0;
    float* state = a.S + ((long long)a.seg_slot[seg] * d.H + h) * kp * vp + c;
    float4 S[NR ? NR : 1];
    if (NR > 0)
#pragma unroll
        for (int i = 0; i < NR; ++i) {
            const int r = rg + i * groups;
            S[i] = on && r < kp && !fresh ? *reinterpret_cast<const float4*>(state + (long long)r * vp) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
    chain_wait();
    const int t = a.seg_start[seg];
    const T* row = static_cast<const T*>(a.qkv) + (long long)t * d.conv_cols();
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
    float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
    auto take = [&](int r, const float4& s) {
        const float k = ks[r], q = qs[r];
        ak.x = fmaf(s.x, k, ak.x); ak.y = fmaf(s.y, k, ak.y); ak.z = fmaf(s.z, k, ak.z); ak.w = fmaf(s.w, k, ak.w);
        aq.x = fmaf(s.x, q, aq.x); aq.y = fmaf(s.y, q, aq.y); aq.z = fmaf(s.z, q, aq.z); aq.w = fmaf(s.w, q, aq.w);
    };
    if (on) {
        if (NR > 0) {
#pragma unroll
            for (int i = 0; i < NR; ++i)
                if (rg + i * groups < kp) take(rg + i * groups, S[i]);
        } else if (!fresh) {
#pragma unroll 4
            for (int r = rg; r < kp; r += groups) take(r, *reinterpret_cast<const float4*>(state + (long long)r * vp));
        }
        *reinterpret_cast<float4*>(pk + rg * vp + c) = ak;
        *reinterpret_cast<float4*>(pq + rg * vp + c) = aq;
    }
    __syncthreads();
    const float nq = DELTA ? a.q_scale / sqrtf(tot[0] + UNIT_EPS) : 1.0f, nk = DELTA ? 1.0f / sqrtf(tot[1] + UNIT_EPS) : 1.0f;
    const float beta = DELTA ? rec_sigmoid(tot[3]) : 1.0f;
    const float gt = DELTA ? expf(a.A[h] * rec_softplus(tot[4] + a.dt_bias[h])) : a.decay[h];
    const float kq = tot[2] * nk * nq;
    // one thread per column: fold the row groups, the new value u and the output
    for (int j = tid; j < vp; j += RT_THREADS) {
        float sk = 0.0f, sq = 0.0f;
        for (int r = 0; r < groups; ++r) { sk += pk[r * vp + j]; sq += pq[r * vp + j]; }
        float u = to_f32(row[2 * d.G * kp + h * vp + j]);
        if (DELTA) u = beta * (u - gt * nk * sk);
        os[j] = fmaf(kq, u, gt * nq * sq);
        pk[j] = u * nk;  // (row group 0 of this column has been read)
    }
    __syncthreads();
    if (on) {
        const float4 u = *reinterpret_cast<const float4*>(pk + c);
        auto put = [&](int r, float4 s) {
            const float k = ks[r];
            s.x = fmaf(k, u.x, gt * s.x); s.y = fmaf(k, u.y, gt * s.y); s.z = fmaf(k, u.z, gt * s.z); s.w = fmaf(k, u.w, gt * s.w);
            *reinterpret_cast<float4*>(state + (long long)r * vp) = s;
        };
        if (NR > 0) {
#pragma unroll
            for (int i = 0; i < NR; ++i)
                if (rg + i * groups < kp) put(rg + i * groups, S[i]);
        } else {
#pragma unroll 4
            for (int r = rg; r < kp; r += groups)
                put(r, fresh ? make_float4(0.f, 0.f, 0.f, 0.f) : *reinterpret_cast<const float4*>(state + (long long)r * vp));
        }
    }
    T* out = static_cast<T*>(a.out) + (long long)t * d.H * vp + h * vp;
    if (!DELTA) {
        for (int j = tid; j < vp; j += RT_THREADS) out[j] = from_f32<T>(os[j]);
        return;
    }
    float ss = 0.0f;
    for (int j = tid; j < vp; j += RT_THREADS) ss = fmaf(os[j], os[j], ss);
    ss = warp_sum(ss);
    if (lane == 0) red[warp][0] = ss;
    __syncthreads();
    ss = 0.0f;
#pragma unroll
    for (int w = 0; w < RT_THREADS / 32; ++w) ss += red[w][0];
    const float rms = sqrtf(ss / (float)d.dv + a.eps);
    const T* z = static_cast<const T*>(a.z) + (long long)t * d.raw_cols() + h * vp;
    for (int j = tid; j < vp; j += RT_THREADS) {
        const float zv = to_f32(z[j]);
        out[j] = from_f32<T>(os[j] / rms * a.norm[j] * (zv * rec_sigmoid(zv)));
    }
}

// ---- norm and gate of the output ----------------------------------------------------------------------------------
// PER_HEAD: every head by itself, weight [vp], gate silu(z); otherwise all heads together, weight [H vp], gate sigmoid(z).
// In place.  One CTA per token.
template <typename T, bool PER_HEAD>
__global__ void __launch_bounds__(256) rec_norm_kernel(T* __restrict__ o, const T* __restrict__ z, long long z_pitch, const float* __restrict__ gain,
                                                       float eps, int H, int dv, int vp) {
    __shared__ float red[8];
    chain_trigger();
    chain_wait();
    T* row = o + (long long)blockIdx.x * H * vp;
    const T* zr = z + blockIdx.x * z_pitch;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (PER_HEAD) {
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
                store_f32x2(row + h * vp + j, a / rms * gain[j] * (za * rec_sigmoid(za)), b / rms * gain[j + 1] * (zb * rec_sigmoid(zb)));
            }
        }
        return;
    }
    const int n = H * vp;
    float ss = 0.0f;
    for (int j = threadIdx.x * 8; j < n; j += 2048) {
        float v[8];
        load_f32x8(row + j, v);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss = fmaf(v[e], v[e], ss);
    }
    ss = warp_sum(ss);
    if (lane == 0) red[warp] = ss;
    __syncthreads();
    ss = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) ss += red[w];
    const float rms = sqrtf(ss / (float)(H * dv) + eps);
    for (int j = threadIdx.x * 8; j < n; j += 2048) {
        float v[8], zv[8], gv[8];
        load_f32x8(row + j, v);
        load_f32x8(zr + j, zv);
        load_f32x8(gain + j, gv);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[e] = v[e] / rms * gv[e] * rec_sigmoid(zv[e]);
        store_f32x8(row + j, v);
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
    JSM_CUDA_CHECK(d.delta ? go(rec_norm_kernel<T, true>) : go(rec_norm_kernel<T, false>));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

bool rec_usable(const RecDims& d) { return d.dk <= 256 && d.dv <= 1024; }

jsm_status rec_scan_launch(bool f32, const RecDims& d, const RecWeights& w, const RecState& s, float eps, const StepTokens& tk, const void* raw,
                           const void* qkv, const float* ba, void* out, cudaStream_t st) {
    if (!rec_usable(d)) JSM_FAIL(JSM_UNSUPPORTED, "linear recurrence: heads of %d / %d components (at most 256 / 1024)", d.dk, d.dv);
    RecArgs a = rec_args(f32, d, w, s, tk, raw, qkv, out, eps);
    a.ba = ba;
    jsm_status r = f32 ? (d.delta ? scan_sized<float, true>(a, d, tk.n_segs, st) : scan_sized<float, false>(a, d, tk.n_segs, st))
                       : (d.delta ? scan_sized<__nv_bfloat16, true>(a, d, tk.n_segs, st) : scan_sized<__nv_bfloat16, false>(a, d, tk.n_segs, st));
    if (r != JSM_OK) return r;
    return f32 ? norm_typed<float>(d, a, tk.T, st) : norm_typed<__nv_bfloat16>(d, a, tk.T, st);
}

template <typename T, int NR, bool DELTA>
static jsm_status step_go(const RecArgs& a, const RecDims& d, int lpr, int n_segs, cudaStream_t st) {
    const size_t smem = sizeof(float) * (2 * d.kp() + 2 * (size_t)(RT_THREADS / lpr) * d.vp() + d.vp());
    JSM_CUDA_CHECK(launch_chained(rec_step_kernel<T, NR, DELTA>, dim3(d.H, n_segs), dim3(RT_THREADS), smem, st, a, d, lpr));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
template <typename T, bool DELTA>
static jsm_status step_sized(const RecArgs& a, const RecDims& d, int n_segs, cudaStream_t st) {
    int lpr = 1;
    while (lpr * 4 < d.vp()) lpr *= 2;
    const int groups = RT_THREADS / lpr, nr = (d.kp() + groups - 1) / groups;
    return nr <= 1 ? step_go<T, 1, DELTA>(a, d, lpr, n_segs, st) : nr <= 2 ? step_go<T, 2, DELTA>(a, d, lpr, n_segs, st)
         : nr <= 4 ? step_go<T, 4, DELTA>(a, d, lpr, n_segs, st) : nr <= 8 ? step_go<T, 8, DELTA>(a, d, lpr, n_segs, st)
         : nr <= 16 ? step_go<T, 16, DELTA>(a, d, lpr, n_segs, st) : step_go<T, 0, DELTA>(a, d, lpr, n_segs, st);
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
