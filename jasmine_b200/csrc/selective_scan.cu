// Selective scan (Mamba) with its short causal convolution, over segments of consecutive tokens of many sequences.
//
//   xc = silu(conv(x) + b)                              (per channel, `taps` inputs back)
//   S[c, n] <- exp(dt_c A[c, n]) S[c, n] + dt_c xc_c B_n      dt_c = softplus(dt_raw_c + dt_b_c)
//   y_c = (sum_n S[c, n] C_n + D_c xc_c) * silu(z_c)
//
// The recurrent state S and everything that enters it is fp32; x, z and y are activations (bf16 or f32).  A sequence's
// state lives in a slot: S and the last taps - 1 inputs of the convolution.  A segment that starts at position 0 starts from
// zeros whatever the slot holds, so a slot needs no clearing when a new sequence takes it.
//
// Prompts: a CTA owns 16 channels of one segment and walks its tokens in tiles of 32 that cp.async brings into a two-stage
// ring; eight threads share a channel's states, so that the chain of dependent steps is one FMA per state and the partial
// sums of eight tokens are exchanged with seven shuffles.  Decode: one thread per channel and sequence, eight sequences per
// CTA; the states are requested first and arrive while the step sizes (a small projection) are computed.
//
// Layout of S and A: planes of four states, [plane][channel][4], so that neighbouring threads - channels - read neighbouring
// 16-byte vectors.
#include "decoder_ops.cuh"
#include "mma_utils.cuh"
#include "tc_utils.cuh"
#include <math.h>
#include <algorithm>

namespace jsm {

using tc::smem_u32;

constexpr int SC_CH = 16;       // channels per CTA
constexpr int SC_SUB = 8;       // threads per channel (prompts)
constexpr int SC_THREADS = SC_CH * SC_SUB;
constexpr int SC_TT = 32;       // tokens per tile
constexpr int SC_YP = SC_CH + 4;  // pitch of the output tile (floats)
constexpr int ST_WARPS = 4;     // decode step: a warp per sequence
constexpr int ST_CH = 32;       // channels per CTA: a lane each
constexpr int ST_THREADS = ST_CH * ST_WARPS;
constexpr int ST_BB = 8;        // sequences per CTA
__host__ __device__ inline long long plane_index(int n, int c, int ip) { return ((long long)(n >> 2) * ip + c) * 4 + (n & 3); }

__device__ __forceinline__ float softplus_f(float x) { return x > 20.0f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float silu_f(float x) { return x / (1.0f + expf(-x)); }
template <typename T>
__device__ __forceinline__ float decay(float x);  // e^x for x <= 0
template <>
__device__ __forceinline__ float decay<float>(float x) { return expf(x); }
template <>
__device__ __forceinline__ float decay<__nv_bfloat16>(float x) { return fast_ex2(LOG2E * x); }
// the forms of a bf16 model: fp32 arithmetic with the fast exponential and logarithm; ln(1 + e) by its series where 1 + e
// would round e away
template <typename T>
__device__ __forceinline__ float softplus_t(float x) {
    if constexpr (sizeof(T) == 4) return softplus_f(x);
    const float e = fast_ex2(LOG2E * x);
    const float series = e * (1.0f - e * (0.5f - e * (0.33333333f - e * (0.25f - e * 0.2f))));
    return x > 20.0f ? x : x < -3.0f ? series : __logf(1.0f + e);
}
template <typename T>
__device__ __forceinline__ float silu_t(float x) {
    if constexpr (sizeof(T) == 4) return silu_f(x);
    return x * fast_rcp(1.0f + fast_ex2(-LOG2E * x));
}

template <typename T>
struct Vec8;
template <>
struct Vec8<float> {
    struct Raw { float4 a, b; };
    __device__ static Raw fetch(const float* p) { return Raw{reinterpret_cast<const float4*>(p)[0], reinterpret_cast<const float4*>(p)[1]}; }
    __device__ static void widen(const Raw& r, float (&v)[8]) {
        v[0] = r.a.x; v[1] = r.a.y; v[2] = r.a.z; v[3] = r.a.w; v[4] = r.b.x; v[5] = r.b.y; v[6] = r.b.z; v[7] = r.b.w;
    }
    __device__ static void load(const float* p, float (&v)[8]) {
        const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    __device__ static void store(float* p, const float (&v)[8]) {
        reinterpret_cast<float4*>(p)[0] = make_float4(v[0], v[1], v[2], v[3]);
        reinterpret_cast<float4*>(p)[1] = make_float4(v[4], v[5], v[6], v[7]);
    }
};
template <>
struct Vec8<__nv_bfloat16> {
    using Raw = uint4;
    __device__ static Raw fetch(const __nv_bfloat16* p) { return *reinterpret_cast<const uint4*>(p); }
    __device__ static void load(const __nv_bfloat16* p, float (&v)[8]) { widen(fetch(p), v); }
    __device__ static void widen(const uint4& w, float (&v)[8]) {
        v[0] = bf16lo(w.x); v[1] = bf16hi(w.x); v[2] = bf16lo(w.y); v[3] = bf16hi(w.y);
        v[4] = bf16lo(w.z); v[5] = bf16hi(w.z); v[6] = bf16lo(w.w); v[7] = bf16hi(w.w);
    }
    __device__ static void store(__nv_bfloat16* p, const float (&v)[8]) {
        uint4 w;
        w.x = pack_bf16x2(v[0], v[1]); w.y = pack_bf16x2(v[2], v[3]); w.z = pack_bf16x2(v[4], v[5]); w.w = pack_bf16x2(v[6], v[7]);
        *reinterpret_cast<uint4*>(p) = w;
    }
};

__device__ __forceinline__ void load4(const float* p, float (&v)[4]) {
    const float4 a = *reinterpret_cast<const float4*>(p);
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load4(const __nv_bfloat16* p, float (&v)[4]) {
    const uint2 a = *reinterpret_cast<const uint2*>(p);
    v[0] = bf16lo(a.x); v[1] = bf16hi(a.x); v[2] = bf16lo(a.y); v[3] = bf16hi(a.y);
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
    *reinterpret_cast<uint2*>(p) = make_uint2(pack_bf16x2(v[0], v[1]), pack_bf16x2(v[2], v[3]));
}

// ---- convolution --------------------------------------------------------------------------------------------------
// A thread owns 8 channels of CONV_TOK consecutive tokens; TAPS 0: taps is only known at run time.  carry: every segment is
// one token, and the state moves on by it here (otherwise the scan does that, once every CTA has read the old state)
constexpr int CONV_TOK = 8;
template <typename T, int TAPS>
__global__ void __launch_bounds__(256, 2) scan_conv_kernel(const T* __restrict__ xz, long long pitch, T* __restrict__ xc, T* state,
                                                        const float* __restrict__ w, const float* __restrict__ b,
                                                        const int32_t* __restrict__ seg_start, const int32_t* __restrict__ seg_len,
                                                        const int32_t* __restrict__ seg_pos0, const int32_t* __restrict__ seg_slot, int ip,
                                                        int taps_rt, int carry) {
    chain_trigger();
    chain_wait();
    const int taps = TAPS ? TAPS : taps_rt;
    const int seg = blockIdx.y, vec = ip / 8;
    const int start = seg_start[seg], len = seg_len[seg], pos0 = seg_pos0[seg];
    const long long i = (long long)blockIdx.x * 256 + threadIdx.x;
    const int c = (int)(i % vec) * 8, j0 = (int)(i / vec) * CONV_TOK;
    if (j0 >= len) return;
    T* st = state + (long long)seg_slot[seg] * (taps - 1) * ip + c;
    // input of the segment's token j (negative: before the segment)
    auto input = [&](int j, float (&v)[8]) {
        if (j >= 0) Vec8<T>::load(xz + (start + j) * pitch + c, v);
        else if (pos0 + j >= 0) Vec8<T>::load(st + (long long)(taps - 1 + j) * ip, v);
        else
            for (int e = 0; e < 8; ++e) v[e] = 0.0f;
    };
    float bias[8];
    if (b) Vec8<float>::load(b + c, bias);
    else
#pragma unroll
        for (int e = 0; e < 8; ++e) bias[e] = 0.0f;
    const int j1 = min(len, j0 + CONV_TOK);
    if constexpr (TAPS > 0) {
        // all the thread's inputs are requested before the first is used
        typename Vec8<T>::Raw raw[CONV_TOK];
#pragma unroll
        for (int u = 0; u < CONV_TOK; ++u)
            if (j0 + u < j1) raw[u] = Vec8<T>::fetch(xz + (start + j0 + u) * pitch + c);
        float win[TAPS][8], wt[TAPS][8];
#pragma unroll
        for (int k = 0; k < TAPS; ++k) Vec8<float>::load(w + (long long)k * ip + c, wt[k]);
#pragma unroll
        for (int k = 0; k + 1 < TAPS; ++k) input(j0 - TAPS + 1 + k, win[k + 1]);
#pragma unroll
        for (int u = 0; u < CONV_TOK; ++u) {
            const int j = j0 + u;
            if (j >= j1) break;
#pragma unroll
            for (int k = 0; k + 1 < TAPS; ++k)
#pragma unroll
                for (int e = 0; e < 8; ++e) win[k][e] = win[k + 1][e];
            Vec8<T>::widen(raw[u], win[TAPS - 1]);
            float o[8];
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                float a = bias[e];
#pragma unroll
                for (int k = 0; k < TAPS; ++k) a = fmaf(wt[k][e], win[k][e], a);
                o[e] = silu_t<T>(a);
            }
            Vec8<T>::store(xc + (long long)(start + j) * ip + c, o);
        }
        if (carry)  // one token per segment: this thread has read all there is to read of its channels' state
#pragma unroll
            for (int k = 0; k + 1 < TAPS; ++k) Vec8<T>::store(st + (long long)k * ip, win[k + 1]);
    } else {
        for (int j = j0; j < j1; ++j) {
            float o[8];
            for (int e = 0; e < 8; ++e) o[e] = bias[e];
            for (int k = 0; k < taps; ++k) {
                float v[8], wk[8];
                input(j - taps + 1 + k, v);
                Vec8<float>::load(w + (long long)k * ip + c, wk);
#pragma unroll
                for (int e = 0; e < 8; ++e) o[e] = fmaf(wk[e], v[e], o[e]);
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) o[e] = silu_t<T>(o[e]);
            Vec8<T>::store(xc + (long long)(start + j) * ip + c, o);
        }
        if (carry)
            for (int k = 0; k + 1 < taps; ++k) {
                float v[8];
                input(k + 2 - taps, v);  // ascending: an entry is read before a later one takes its place
                Vec8<T>::store(st + (long long)k * ip, v);
            }
    }
}

// the last taps - 1 inputs after the segment: entry k is the input taps - 1 - k tokens before the next one.  One thread per
// channel, ascending k: an entry taken from the old state lies behind every entry already written.
template <typename T>
__device__ __forceinline__ void carry_conv_state(T* state, const T* __restrict__ xz, long long pitch, int c, int ip, int taps, int start, int len,
                                                 int pos0) {
    for (int k = 0; k + 1 < taps; ++k) {
        const int j = len - (taps - 1) + k;
        T v = from_f32<T>(0.0f);
        if (j >= 0) v = xz[(start + j) * pitch + c];
        else if (pos0 + j >= 0) v = state[(long long)(k + len) * ip + c];
        state[(long long)k * ip + c] = v;
    }
}

template <int NS>
__device__ __forceinline__ void lds_vec(const float* p, float (&v)[NS]) {
    if constexpr (NS % 4 == 0) {
#pragma unroll
        for (int i = 0; i < NS; i += 4) {
            const float4 a = *reinterpret_cast<const float4*>(p + i);
            v[i] = a.x; v[i + 1] = a.y; v[i + 2] = a.z; v[i + 3] = a.w;
        }
    } else if constexpr (NS % 2 == 0) {
#pragma unroll
        for (int i = 0; i < NS; i += 2) {
            const float2 a = *reinterpret_cast<const float2*>(p + i);
            v[i] = a.x; v[i + 1] = a.y;
        }
    } else {
#pragma unroll
        for (int i = 0; i < NS; ++i) v[i] = p[i];
    }
}

// ---- scan of prompts ----------------------------------------------------------------------------------------------
__host__ __device__ inline int scan_nb(int np, int ns) { return np > SC_SUB * ns ? np : SC_SUB * ns; }  // B / C columns per tile row
template <typename T>
static size_t scan_smem(int np, int ns) {
    return 2 * (size_t)SC_TT * SC_CH * (2 * sizeof(T) + 4) + 2 * (size_t)SC_TT * 2 * scan_nb(np, ns) * 4 + (size_t)SC_TT * SC_YP * 4 +
           (size_t)SC_TT * SC_CH * 16;
}

struct ScanArgs {
    const float *A, *D, *dt_b, *proj, *dt_raw;
    const void *xz, *xc, *dt_w;
    void *y, *conv;
    float* S;
    const int32_t *seg_start, *seg_len, *seg_pos0, *seg_slot;
    int ip, np, rp, state, taps, n_segs;
};

template <typename T, int NS>
__global__ void __launch_bounds__(SC_THREADS) scan_kernel(ScanArgs a) {
    extern __shared__ __align__(16) uint8_t sc_dyn[];
    const int nb = scan_nb(a.np, NS);
    T* xs = reinterpret_cast<T*>(sc_dyn);                                   // 2 x [TT][CH]
    T* zs = xs + 2 * SC_TT * SC_CH;                                         // 2 x [TT][CH]
    float* dts = reinterpret_cast<float*>(zs + 2 * SC_TT * SC_CH);          // 2 x [TT][CH]
    float* bc = dts + 2 * SC_TT * SC_CH;                                    // 2 x [TT][B: nb | C: nb]
    float* ys = bc + 2 * SC_TT * 2 * nb;                                    // [TT][YP]
    float4* dd = reinterpret_cast<float4*>(ys + SC_TT * SC_YP);             // [TT][CH]: dt, dt, dt x, dt x
    constexpr bool PAIRS = sizeof(T) == 2 && NS % 2 == 0;                   // bf16 models: states in pairs, base-2 exponentials
    chain_trigger();
    const int tid = threadIdx.x, ch = tid / SC_SUB, sub = tid % SC_SUB;
    const int c0 = blockIdx.x * SC_CH, c = c0 + ch;
    const bool live = c < a.ip;
    float A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int n = sub * NS + i;
        A[i] = (live && n < a.state) ? a.A[plane_index(n, c, a.ip)] : 0.0f;
        if (PAIRS) A[i] *= LOG2E;
    }
    for (int i = tid; i < 2 * SC_TT * 2 * nb; i += SC_THREADS) bc[i] = 0.0f;  // columns behind np stay zero
    __syncthreads();
    chain_wait();
    const int seg = blockIdx.y;
    const int start = a.seg_start[seg], len = a.seg_len[seg], pos0 = a.seg_pos0[seg], slot = a.seg_slot[seg];
    float* state = a.S + (long long)slot * a.ip * a.np;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int n = sub * NS + i;
        S[i] = (live && n < a.state && pos0 > 0) ? state[plane_index(n, c, a.ip)] : 0.0f;
    }
    const int pc = a.rp + 2 * a.np;
    const T* xz = static_cast<const T*>(a.xz);
    const T* xc = static_cast<const T*>(a.xc);
    auto load_tile = [&](int t0, int stage) {
        constexpr int EV = 16 / sizeof(T), XV = SC_CH / EV;  // elements per vector, vectors per row
        for (int i = tid; i < SC_TT * XV; i += SC_THREADS) {
            const int r = i / XV, v = (i % XV) * EV;
            const bool ok = t0 + r < len && c0 + v < a.ip;
            const long long t = start + (ok ? t0 + r : 0);
            const int cc = ok ? c0 + v : 0;
            cp_async16(smem_u32(xs + (stage * SC_TT + r) * SC_CH + v), xc + t * a.ip + cc, ok);
            cp_async16(smem_u32(zs + (stage * SC_TT + r) * SC_CH + v), xz + t * 2 * a.ip + a.ip + cc, ok);
        }
        for (int i = tid; i < SC_TT * (SC_CH / 4); i += SC_THREADS) {
            const int r = i / (SC_CH / 4), v = (i % (SC_CH / 4)) * 4;
            const bool ok = t0 + r < len && c0 + v < a.ip;
            cp_async16(smem_u32(dts + (stage * SC_TT + r) * SC_CH + v), a.dt_raw + (long long)(start + (ok ? t0 + r : 0)) * a.ip + (ok ? c0 + v : 0), ok);
        }
        const int bv = a.np / 4;
        for (int i = tid; i < SC_TT * 2 * bv; i += SC_THREADS) {
            const int r = i / (2 * bv), v = i % (2 * bv);
            const bool ok = t0 + r < len;
            const float* src = a.proj + (long long)(start + (ok ? t0 + r : 0)) * pc + a.rp + v * 4;
            cp_async16(smem_u32(bc + ((stage * SC_TT + r) * 2 + (v >= bv)) * nb + (v % bv) * 4), src, ok);
        }
    };
    load_tile(0, 0);
    cp_async_commit();
    // every pass over a tile gives a thread the same channels: their constants stay in registers
    static_assert(SC_THREADS % SC_CH == 0 && SC_TT * SC_CH == SC_THREADS * 4, "four elements of a tile per thread");
    const float bias = c0 + (tid & (SC_CH - 1)) < a.ip ? a.dt_b[c0 + (tid & (SC_CH - 1))] : 0.0f;
    const int ov = (tid & (SC_CH / 4 - 1)) * 4, orow = tid / (SC_CH / 4);  // output pass: four channels of one token
    const bool olive = c0 + ov < a.ip;
    const float4 Dv = olive ? *reinterpret_cast<const float4*>(a.D + c0 + ov) : make_float4(0.f, 0.f, 0.f, 0.f);
    const int nt = (len + SC_TT - 1) / SC_TT;
    for (int it = 0; it < nt; ++it) {
        const int stage = it & 1, t0 = it * SC_TT, n = min(SC_TT, len - t0);
        if (it + 1 < nt) load_tile(t0 + SC_TT, stage ^ 1);
        cp_async_commit();
        cp_async_wait<1>();
        __syncthreads();
        const float* dt = dts + stage * SC_TT * SC_CH;
        const T* x = xs + stage * SC_TT * SC_CH;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int i = u * SC_THREADS + tid;
            // a step size of zero leaves the state as it is: the rows behind the segment (and channels behind the last)
            const float d = i / SC_CH < n ? softplus_t<T>(dt[i] + bias) : 0.0f, dx = d * to_f32(x[i]);
            dd[i] = make_float4(d, d, dx, dx);
        }
        __syncthreads();
        const float* bt = bc + stage * SC_TT * 2 * nb + sub * NS;
#pragma unroll 1
        for (int t8 = 0; t8 < n; t8 += 8) {
            float y[8];
#pragma unroll
            for (int u = 0; u < 8; ++u) {
                const int t = t8 + u;
                if constexpr (PAIRS) {
                    const ulonglong2 w = *reinterpret_cast<const ulonglong2*>(dd + t * SC_CH + ch);  // (dt, dt), (dt x, dt x)
                    const uint64_t* B = reinterpret_cast<const uint64_t*>(bt + t * 2 * nb);
                    const uint64_t* C = reinterpret_cast<const uint64_t*>(bt + t * 2 * nb + nb);
                    uint64_t acc = 0;
#pragma unroll
                    for (int i = 0; i < NS / 2; ++i) {
                        float e0, e1;
                        f2_unpack(f2_mul(w.x, f2_pack(A[2 * i], A[2 * i + 1])), e0, e1);
                        const uint64_t s2 = f2_fma(f2_pack(fast_ex2(e0), fast_ex2(e1)), f2_pack(S[2 * i], S[2 * i + 1]), f2_mul(w.y, B[i]));
                        f2_unpack(s2, S[2 * i], S[2 * i + 1]);
                        acc = i == 0 ? f2_mul(s2, C[i]) : f2_fma(s2, C[i], acc);
                    }
                    float lo, hi;
                    f2_unpack(acc, lo, hi);
                    y[u] = lo + hi;
                } else {
                    const float4 w = dd[t * SC_CH + ch];
                    float B[NS], C[NS];
                    lds_vec<NS>(bt + t * 2 * nb, B);
                    lds_vec<NS>(bt + t * 2 * nb + nb, C);
                    float acc = 0.0f;
#pragma unroll
                    for (int i = 0; i < NS; ++i) {
                        S[i] = fmaf(decay<T>(w.x * A[i]), S[i], w.z * B[i]);
                        acc = fmaf(S[i], C[i], acc);
                    }
                    y[u] = acc;
                }
            }
            // eight partial sums on each of eight lanes -> lane `sub` holds the sum of token t8 + sub
            float k4[4], k2[2];
#pragma unroll
            for (int u = 0; u < 4; ++u) k4[u] = ((sub & 4) ? y[4 + u] : y[u]) + __shfl_xor_sync(0xffffffffu, (sub & 4) ? y[u] : y[4 + u], 4);
#pragma unroll
            for (int u = 0; u < 2; ++u) k2[u] = ((sub & 2) ? k4[2 + u] : k4[u]) + __shfl_xor_sync(0xffffffffu, (sub & 2) ? k4[u] : k4[2 + u], 2);
            const float k = ((sub & 1) ? k2[1] : k2[0]) + __shfl_xor_sync(0xffffffffu, (sub & 1) ? k2[0] : k2[1], 1);
            ys[(t8 + sub) * SC_YP + ch] = k;
        }
        __syncthreads();
        const T* z = zs + stage * SC_TT * SC_CH;
        if (orow < n && olive) {
            float xv[4], zv[4], o[4];
            load4(x + orow * SC_CH + ov, xv);
            load4(z + orow * SC_CH + ov, zv);
            const float4 yv = *reinterpret_cast<const float4*>(ys + orow * SC_YP + ov);
            o[0] = fmaf(Dv.x, xv[0], yv.x) * silu_t<T>(zv[0]); o[1] = fmaf(Dv.y, xv[1], yv.y) * silu_t<T>(zv[1]);
            o[2] = fmaf(Dv.z, xv[2], yv.z) * silu_t<T>(zv[2]); o[3] = fmaf(Dv.w, xv[3], yv.w) * silu_t<T>(zv[3]);
            store4(static_cast<T*>(a.y) + (long long)(start + t0 + orow) * a.ip + c0 + ov, o);
        }
        __syncthreads();
    }
    if (live)
#pragma unroll
        for (int i = 0; i < NS; ++i)
            if (sub * NS + i < a.state) state[plane_index(sub * NS + i, c, a.ip)] = S[i];
    if (tid < SC_CH && c0 + tid < a.ip)
        carry_conv_state(static_cast<T*>(a.conv) + (long long)slot * (a.taps - 1) * a.ip, xz, 2 * a.ip, c0 + tid, a.ip, a.taps, start, len,
                            pos0);
}

// ---- decode step --------------------------------------------------------------------------------------------------
// One token of up to 8 sequences and 32 channels per CTA: lane = channel, a warp takes two sequences; the convolution has
// already moved its state on.  The step sizes of the 32 channels x 8 sequences are one small product: bf16 models take it on
// the tensor cores (weights as the 16-row operand, two tiles of channels x two halves of the rank over the four warps).
// NP: planes of four states kept in registers, requested before the step sizes are known; 0 = any number, read when needed.
template <typename T, int NP>
__global__ void __launch_bounds__(ST_THREADS) scan_step_kernel(ScanArgs a) {
    extern __shared__ __align__(16) float st_dyn[];  // bf16: [8][B: np | C: np]; f32: [8][proj columns]
    __shared__ float dts[2][ST_CH][9];
    constexpr bool MMA = sizeof(T) == 2;
    constexpr int R = ST_BB / ST_WARPS;  // sequences per warp
    chain_trigger();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int c0 = blockIdx.x * ST_CH, c = c0 + lane, cl = min(c, a.ip - 1);
    const bool live = c < a.ip;
    const int s0 = blockIdx.y * ST_BB, nb = min(ST_BB, a.n_segs - s0);
    const int pc = a.rp + 2 * a.np, off = MMA ? a.rp : 0, sc = pc - off;  // columns of proj that go to shared memory
    const int planes = a.np / 4;
    const float4* Ap = reinterpret_cast<const float4*>(a.A) + cl;
    float4 A[NP ? NP : 1];
    if (NP > 0)
#pragma unroll
        for (int i = 0; i < NP; ++i) A[i] = i < planes ? Ap[(long long)i * a.ip] : make_float4(0.f, 0.f, 0.f, 0.f);
    const float bias = a.dt_b[cl], dv = a.D[cl];
    chain_wait();
    for (int i = tid; i < nb * (sc / 4); i += ST_THREADS) {
        const int b = i / (sc / 4), v = i % (sc / 4);
        cp_async16(smem_u32(st_dyn + i * 4), a.proj + (long long)a.seg_start[s0 + b] * pc + off + v * 4, true);
    }
    cp_async_commit();
    float4 S[R][NP ? NP : 1];
    float4* Sp[R];
    bool fresh[R];
    int tok[R];
    T xv[R], zv[R];
#pragma unroll
    for (int q = 0; q < R; ++q) {
        const int sg = s0 + min(q * ST_WARPS + warp, nb - 1);
        tok[q] = a.seg_start[sg];
        fresh[q] = a.seg_pos0[sg] == 0;
        Sp[q] = reinterpret_cast<float4*>(a.S + (long long)a.seg_slot[sg] * a.ip * a.np) + cl;
        if (NP > 0)
#pragma unroll
            for (int i = 0; i < NP; ++i)
                S[q][i] = (i < planes && !fresh[q]) ? Sp[q][(long long)i * a.ip] : make_float4(0.f, 0.f, 0.f, 0.f);
        xv[q] = static_cast<const T*>(a.xc)[(long long)tok[q] * a.ip + cl];
        zv[q] = static_cast<const T*>(a.xz)[(long long)tok[q] * 2 * a.ip + a.ip + cl];
    }
    if constexpr (MMA) {
        const int mt = warp & 1, kh = warp >> 1, g = lane >> 2, kq = (lane & 3) * 8;
        const int n_blk = (a.rp + 31) / 32, b0 = kh ? (n_blk + 1) / 2 : 0, b1 = kh ? n_blk : (n_blk + 1) / 2;
        const int r0 = c0 + mt * 16 + g;
        const __nv_bfloat16* w0 = static_cast<const __nv_bfloat16*>(a.dt_w) + (long long)min(r0, a.ip - 1) * a.rp;
        const __nv_bfloat16* w1 = static_cast<const __nv_bfloat16*>(a.dt_w) + (long long)min(r0 + 8, a.ip - 1) * a.rp;
        const float* p = a.proj + (long long)a.seg_start[s0 + min(g, nb - 1)] * pc;
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll 4
        for (int blk = b0; blk < b1; ++blk) {
            const int k = blk * 32 + kq;
            uint4 x = make_uint4(0, 0, 0, 0), y = x;
            float4 u = make_float4(0.f, 0.f, 0.f, 0.f), v = u;
            if (k < a.rp) {
                x = __ldg(reinterpret_cast<const uint4*>(w0 + k));
                y = __ldg(reinterpret_cast<const uint4*>(w1 + k));
                u = reinterpret_cast<const float4*>(p + k)[0];
                v = reinterpret_cast<const float4*>(p + k)[1];
            }
            const uint32_t a0[4] = {x.x, y.x, x.y, y.y}, a1[4] = {x.z, y.z, x.w, y.w};
            mma_16816(acc, a0, pack_bf16x2(u.x, u.y), pack_bf16x2(u.z, u.w));
            mma_16816(acc, a1, pack_bf16x2(v.x, v.y), pack_bf16x2(v.z, v.w));
        }
        float* d = &dts[kh][mt * 16 + g][(lane & 3) * 2];
        d[0] = acc[0]; d[1] = acc[1]; d[8 * 9] = acc[2]; d[8 * 9 + 1] = acc[3];
    }
    cp_async_wait<0>();
    __syncthreads();
#pragma unroll
    for (int q = 0; q < R; ++q) {
        const int b = q * ST_WARPS + warp;
        if (b >= nb) break;
        float raw = 0.0f;
        if constexpr (MMA) {
            raw = dts[0][lane][b] + dts[1][lane][b];
        } else {
            const T* w = static_cast<const T*>(a.dt_w) + (long long)cl * a.rp;
            for (int r = 0; r < a.rp; ++r) raw = fmaf(to_f32(w[r]), st_dyn[b * sc + r], raw);
        }
        const float x = to_f32(xv[q]), dt = softplus_t<T>(raw + bias), dx = dt * x;
        const float4* Bp = reinterpret_cast<const float4*>(st_dyn + b * sc + (a.rp - off));
        const float4* Cp = Bp + planes;
        float y = 0.0f;
        auto plane = [&](int i, const float4& Ai, float4& s) {
            const float4 B = Bp[i], C = Cp[i];
            s.x = fmaf(decay<T>(dt * Ai.x), s.x, dx * B.x); y = fmaf(s.x, C.x, y);
            s.y = fmaf(decay<T>(dt * Ai.y), s.y, dx * B.y); y = fmaf(s.y, C.y, y);
            s.z = fmaf(decay<T>(dt * Ai.z), s.z, dx * B.z); y = fmaf(s.z, C.z, y);
            s.w = fmaf(decay<T>(dt * Ai.w), s.w, dx * B.w); y = fmaf(s.w, C.w, y);
            if (live) Sp[q][(long long)i * a.ip] = s;
        };
        if constexpr (NP > 0) {
#pragma unroll
            for (int i = 0; i < NP; ++i)
                if (i < planes) plane(i, A[i], S[q][i]);
        } else {
#pragma unroll 2
            for (int i = 0; i < planes; ++i) {
                float4 s = fresh[q] ? make_float4(0.f, 0.f, 0.f, 0.f) : Sp[q][(long long)i * a.ip];
                plane(i, Ap[(long long)i * a.ip], s);
            }
        }
        if (live) static_cast<T*>(a.y)[(long long)tok[q] * a.ip + c] = from_f32<T>(fmaf(dv, x, y) * silu_t<T>(to_f32(zv[q])));
    }
}

__global__ void __launch_bounds__(256) scan_dt_operand_kernel(const float* __restrict__ proj, __nv_bfloat16* __restrict__ out, int T, int rp, int pc) {
    chain_trigger();
    chain_wait();
    const int vec = rp / 8;
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < (long long)T * vec; i += (long long)gridDim.x * 256) {
        const int t = (int)(i / vec), c = (int)(i % vec) * 8;
        float v[8];
        Vec8<float>::load(proj + (long long)t * pc + c, v);
        Vec8<__nv_bfloat16>::store(out + (long long)t * rp + c, v);
    }
}

// ---- launches -----------------------------------------------------------------------------------------------------
template <typename T>
static jsm_status conv_typed(const void* x, long long pitch, int cp, int taps, const float* w, const float* b, void* state, const StepTokens& tk, void* out,
                             bool carry, cudaStream_t st) {
    const long long n = (long long)((tk.max_len + CONV_TOK - 1) / CONV_TOK) * (cp / 8);
    const dim3 grid((unsigned)((n + 255) / 256), tk.n_segs);
    auto go = [&](auto kernel) {
        return launch_chained(kernel, grid, dim3(256), 0, st, (const T*)x, pitch, (T*)out, (T*)state, w, b, tk.seg_start, tk.seg_len, tk.seg_pos0,
                              tk.seg_slot, cp, taps, carry ? 1 : 0);
    };
    JSM_CUDA_CHECK(taps == 1 ? go(scan_conv_kernel<T, 1>) : taps == 2 ? go(scan_conv_kernel<T, 2>) : taps == 3 ? go(scan_conv_kernel<T, 3>)
                   : taps == 4 ? go(scan_conv_kernel<T, 4>) : go(scan_conv_kernel<T, 0>));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

jsm_status short_conv_launch(bool f32, const void* x, long long x_pitch, int cp, int taps, const float* w, const float* bias, void* state,
                             const StepTokens& tk, void* out, bool carry, cudaStream_t st) {
    return f32 ? conv_typed<float>(x, x_pitch, cp, taps, w, bias, state, tk, out, carry, st)
               : conv_typed<__nv_bfloat16>(x, x_pitch, cp, taps, w, bias, state, tk, out, carry, st);
}

jsm_status scan_conv_launch(bool f32, const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz,
                            void* xc, bool carry, cudaStream_t st) {
    return short_conv_launch(f32, xz, 2 * d.ip(), d.ip(), d.taps, w.conv, w.conv_b, s.conv, tk, xc, carry, st);
}

template <typename T>
__global__ void __launch_bounds__(256) conv_carry_kernel(const T* __restrict__ x, long long pitch, T* state, const int32_t* __restrict__ seg_start,
                                                         const int32_t* __restrict__ seg_len, const int32_t* __restrict__ seg_pos0,
                                                         const int32_t* __restrict__ seg_slot, int cp, int taps) {
    chain_trigger();
    chain_wait();
    const int c = blockIdx.x * 256 + threadIdx.x, seg = blockIdx.y;
    if (c < cp) carry_conv_state(state + (long long)seg_slot[seg] * (taps - 1) * cp, x, pitch, c, cp, taps, seg_start[seg], seg_len[seg], seg_pos0[seg]);
}
jsm_status short_conv_carry_launch(bool f32, const void* x, long long x_pitch, int cp, int taps, void* state, const StepTokens& tk, cudaStream_t st) {
    if (taps <= 1) return JSM_OK;
    const dim3 grid((cp + 255) / 256, tk.n_segs);
    if (f32) JSM_CUDA_CHECK(launch_chained(conv_carry_kernel<float>, grid, dim3(256), 0, st, (const float*)x, x_pitch, (float*)state, tk.seg_start, tk.seg_len,
                                           tk.seg_pos0, tk.seg_slot, cp, taps));
    else JSM_CUDA_CHECK(launch_chained(conv_carry_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, (const __nv_bfloat16*)x, x_pitch, (__nv_bfloat16*)state,
                                       tk.seg_start, tk.seg_len, tk.seg_pos0, tk.seg_slot, cp, taps));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

static ScanArgs scan_args(const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz, const void* xc,
                          const float* proj, const float* dt_raw, void* y) {
    ScanArgs a;
    a.A = w.A; a.D = w.D; a.dt_b = w.dt_b; a.proj = proj; a.dt_raw = dt_raw; a.xz = xz; a.xc = xc; a.dt_w = w.dt; a.y = y;
    a.conv = s.conv; a.S = s.S;
    a.seg_start = tk.seg_start; a.seg_len = tk.seg_len; a.seg_pos0 = tk.seg_pos0; a.seg_slot = tk.seg_slot;
    a.ip = d.ip(); a.np = d.np(); a.rp = d.rp(); a.state = d.state; a.taps = d.taps; a.n_segs = tk.n_segs;
    return a;
}

template <typename T, int NS>
static jsm_status scan_go(const ScanArgs& a, cudaStream_t st) {
    static bool attr_done = false;
    if (!attr_done) {
        JSM_CUDA_CHECK(cudaFuncSetAttribute(scan_kernel<T, NS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024));
        attr_done = true;
    }
    JSM_CUDA_CHECK(launch_chained(scan_kernel<T, NS>, dim3((a.ip + SC_CH - 1) / SC_CH, a.n_segs), dim3(SC_THREADS), scan_smem<T>(a.np, NS), st, a));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
template <typename T, int NP>
static jsm_status step_go(const ScanArgs& a, cudaStream_t st) {
    const size_t smem = (size_t)ST_BB * (2 * a.np + (sizeof(T) == 2 ? 0 : a.rp)) * sizeof(float);
    static bool attr_done = false;
    if (!attr_done) {
        JSM_CUDA_CHECK(cudaFuncSetAttribute(scan_step_kernel<T, NP>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
        attr_done = true;
    }
    JSM_CUDA_CHECK(launch_chained(scan_step_kernel<T, NP>, dim3((a.ip + ST_CH - 1) / ST_CH, (a.n_segs + ST_BB - 1) / ST_BB), dim3(ST_THREADS), smem, st, a));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
// the smallest instance whose threads hold a channel's states
template <typename T>
static jsm_status scan_dispatch(const ScanArgs& a, cudaStream_t st) {
    return a.state <= 8 ? scan_go<T, 1>(a, st) : a.state <= 16 ? scan_go<T, 2>(a, st) : a.state <= 24 ? scan_go<T, 3>(a, st)
         : a.state <= 32 ? scan_go<T, 4>(a, st) : a.state <= 64 ? scan_go<T, 8>(a, st) : scan_go<T, 16>(a, st);
}
template <typename T>
static jsm_status step_dispatch(const ScanArgs& a, cudaStream_t st) {
    return a.np <= 8 ? step_go<T, 2>(a, st) : a.np <= 16 ? step_go<T, 4>(a, st) : a.np <= 32 ? step_go<T, 8>(a, st) : step_go<T, 0>(a, st);
}

jsm_status scan_launch(bool f32, const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz,
                       const void* xc, const float* proj, const float* dt_raw, void* y, cudaStream_t st) {
    if (d.state > 128) JSM_FAIL(JSM_UNSUPPORTED, "selective scan: %d states per channel (at most 128)", d.state);
    const ScanArgs a = scan_args(d, w, s, tk, xz, xc, proj, dt_raw, y);
    return f32 ? scan_dispatch<float>(a, st) : scan_dispatch<__nv_bfloat16>(a, st);
}

jsm_status scan_step_launch(bool f32, const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz,
                            const void* xc, const float* proj, void* y, cudaStream_t st) {
    if (d.state > 128) JSM_FAIL(JSM_UNSUPPORTED, "selective scan: %d states per channel (at most 128)", d.state);
    const ScanArgs a = scan_args(d, w, s, tk, xz, xc, proj, nullptr, y);
    return f32 ? step_dispatch<float>(a, st) : step_dispatch<__nv_bfloat16>(a, st);
}

jsm_status scan_dt_operand_launch(const ScanDims& d, const float* proj, void* out, int T, cudaStream_t st) {
    const long long n = (long long)T * (d.rp() / 8);
    JSM_CUDA_CHECK(launch_chained(scan_dt_operand_kernel, dim3((unsigned)std::min<long long>((n + 255) / 256, 148 * 8)), dim3(256), 0, st, proj,
                                  (__nv_bfloat16*)out, T, d.rp(), d.proj_cols()));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

}  // namespace jsm
