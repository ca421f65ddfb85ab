// Token-level kernels of the decoder: embedding gather, fused residual-add + norm.
// None of these exist in the reference (its inputs are real-valued matrices); the
// norm follows the formula of layer_norm_net_t::forward (mat_net_t.hpp:209-225)
// with eps under the square root, RMSNorm drops the mean.
#include "common.cuh"
#include "decoder_ops.cuh"
#include <math.h>
#include <algorithm>

namespace jsm {

template <typename T>
struct VecIO;
template <>
struct VecIO<float> {
    static constexpr int N = 4;
    __device__ static void load(const float* p, float (&v)[4]) {
        float4 t = *reinterpret_cast<const float4*>(p);
        v[0] = t.x; v[1] = t.y; v[2] = t.z; v[3] = t.w;
    }
    __device__ static void store(float* p, const float (&v)[4]) {
        *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]);
    }
};
template <>
struct VecIO<__nv_bfloat16> {
    static constexpr int N = 8;
    __device__ static void load(const __nv_bfloat16* p, float (&v)[8]) {
        uint4 t = *reinterpret_cast<const uint4*>(p);
        v[0] = bf16lo(t.x); v[1] = bf16hi(t.x); v[2] = bf16lo(t.y); v[3] = bf16hi(t.y);
        v[4] = bf16lo(t.z); v[5] = bf16hi(t.z); v[6] = bf16lo(t.w); v[7] = bf16hi(t.w);
    }
    __device__ static void store(__nv_bfloat16* p, const float (&v)[8]) {
        uint4 t;
        t.x = pack_bf16x2(v[0], v[1]); t.y = pack_bf16x2(v[2], v[3]);
        t.z = pack_bf16x2(v[4], v[5]); t.w = pack_bf16x2(v[6], v[7]);
        *reinterpret_cast<uint4*>(p) = t;
    }
};

template <typename T>
__global__ void __launch_bounds__(256) embedding_kernel(const T* __restrict__ table, const T* __restrict__ pos_table,
                                                        const int32_t* __restrict__ ids, const int32_t* __restrict__ positions,
                                                        T* __restrict__ out, int d) {
    constexpr int N = VecIO<T>::N;
    chain_trigger();
    chain_wait();
    const int t = blockIdx.x;
    const long long row = ids[t];
    const long long prow = pos_table ? (positions ? positions[t] : t) : 0;
    for (int c = threadIdx.x * N; c < d; c += 256 * N) {
        float a[N];
        VecIO<T>::load(table + row * d + c, a);
        if (pos_table) {
            float p[N];
            VecIO<T>::load(pos_table + prow * d + c, p);
#pragma unroll
            for (int i = 0; i < N; ++i) a[i] = a[i] + p[i];
        }
        VecIO<T>::store(out + (long long)t * d + c, a);
    }
}

__device__ __forceinline__ float block_sum(float v, float* smem) {
    v = warp_sum(v);
    __syncthreads();
    if ((threadIdx.x & 31) == 0) smem[threadIdx.x >> 5] = v;
    __syncthreads();
    float s = 0.0f;
#pragma unroll
    for (int w = 0; w < 8; ++w) s += smem[w];
    return s;
}

// one CTA per token; the token's features stay in registers between the statistics and the write
template <typename T, int MAXV>
__global__ void __launch_bounds__(256) add_norm_kernel(int kind, const T* __restrict__ h, const T* __restrict__ delta,
                                                       T* __restrict__ h_out, T* __restrict__ y, const float* __restrict__ gain,
                                                       const float* __restrict__ bias, float eps, int d) {
    __shared__ float smem[8];
    constexpr int N = VecIO<T>::N;
    const long long base = (long long)blockIdx.x * d;
    float v[MAXV][N];
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int c = (i * 256 + threadIdx.x) * N;
        if (c < d) {
            VecIO<T>::load(h + base + c, v[i]);
            if (delta) {
                float e[N];
                VecIO<T>::load(delta + base + c, e);
#pragma unroll
                for (int j = 0; j < N; ++j) v[i][j] = v[i][j] + e[j];
                if (sizeof(T) == 2) {  // the residual stream is stored in bf16: normalise what is stored
#pragma unroll
                    for (int j = 0; j < N; ++j) v[i][j] = bf16_bits_to_f32(f32_to_bf16_bits(v[i][j]));
                }
            }
            if (h_out) VecIO<T>::store(h_out + base + c, v[i]);
        } else {
#pragma unroll
            for (int j = 0; j < N; ++j) v[i][j] = 0.0f;
        }
    }
    float mean = 0.0f;
    if (kind == JSM_ROWS_LAYERNORM) {
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < MAXV; ++i)
#pragma unroll
            for (int j = 0; j < N; ++j) s += v[i][j];
        mean = block_sum(s, smem) / (float)d;
    }
    float q = 0.0f;
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int c = (i * 256 + threadIdx.x) * N;
#pragma unroll
        for (int j = 0; j < N; ++j) {
            float dd = v[i][j] - mean;
            v[i][j] = dd;
            q += (c < d) ? dd * dd : 0.0f;
        }
    }
    q = block_sum(q, smem) / (float)d;
    const float sd = sqrtf(q + eps);
#pragma unroll
    for (int i = 0; i < MAXV; ++i) {
        const int c = (i * 256 + threadIdx.x) * N;
        if (c < d) {
            float o[N];
#pragma unroll
            for (int j = 0; j < N; ++j) {
                const float g = gain ? gain[c + j] : 1.0f;
                const float b = (bias && kind == JSM_ROWS_LAYERNORM) ? bias[c + j] : 0.0f;
                o[j] = g * (v[i][j] / sd) + b;
            }
            VecIO<T>::store(y + base + c, o);
        }
    }
}

// ---- decoders whose residual stream is fp32 and whose norms sit on the sublayers' outputs ---------------------------------
template <typename T>
__global__ void __launch_bounds__(256) embed_residual_kernel(const T* __restrict__ table, const int32_t* __restrict__ ids, float* __restrict__ x,
                                                             T* __restrict__ xa, float scale, int wp) {
    constexpr int N = VecIO<T>::N;
    chain_trigger();
    chain_wait();
    const T* src = table + (long long)ids[blockIdx.x] * wp;
    float* dst = x + (long long)blockIdx.x * wp;
    for (int c = threadIdx.x * N; c < wp; c += 256 * N) {
        float v[N];
        VecIO<T>::load(src + c, v);
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] *= scale;
#pragma unroll
        for (int i = 0; i < N; i += 4) *reinterpret_cast<float4*>(dst + c + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
        if (xa) VecIO<T>::store(xa + (long long)blockIdx.x * wp + c, v);
    }
}

// One CTA per token; the sublayer's output y stays in registers between the statistics and the update (MAXV > 0: wp <=
// 2048 * MAXV), or is read twice (MAXV 0).  Padding columns of y and of the gain are zero.
// SUM false: x <- x + norm(y); true: x <- norm(alpha x + y)
template <int MAXV, bool SUM>
__global__ void __launch_bounds__(256) post_norm_add_kernel(const float* __restrict__ y, float* __restrict__ x, const float* __restrict__ gain,
                                                            float eps, float alpha, __nv_bfloat16* __restrict__ xa, int d, int wp) {
    __shared__ float smem[8];
    chain_trigger();
    chain_wait();
    const long long base = (long long)blockIdx.x * wp;
    auto load8 = [](const float* p, float (&v)[8]) {
        const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    };
    float keep[MAXV ? MAXV : 1][8], res[MAXV ? MAXV : 1][8];
    float q = 0.0f;
    if constexpr (MAXV > 0) {
#pragma unroll
        for (int i = 0; i < MAXV; ++i) {
            const int c = (i * 256 + threadIdx.x) * 8;
            if (c < wp) {
                load8(y + base + c, keep[i]);
                load8(x + base + c, res[i]);
                if (SUM)
#pragma unroll
                    for (int e = 0; e < 8; ++e) keep[i][e] = fmaf(alpha, res[i][e], keep[i][e]);
#pragma unroll
                for (int e = 0; e < 8; ++e) q = fmaf(keep[i][e], keep[i][e], q);
            }
        }
    } else {
        for (int c = threadIdx.x * 8; c < wp; c += 2048) {
            float v[8], r[8];
            load8(y + base + c, v);
            if (SUM) {
                load8(x + base + c, r);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = fmaf(alpha, r[e], v[e]);
            }
#pragma unroll
            for (int e = 0; e < 8; ++e) q = fmaf(v[e], v[e], q);
        }
    }
    q = block_sum(q, smem) / (float)d;
    const float rms = sqrtf(q + eps);
    auto update = [&](int c, const float (&v)[8], float (&r)[8]) {
        float g[8];
        load8(gain + c, g);
#pragma unroll
        for (int e = 0; e < 8; ++e) r[e] = SUM ? v[e] / rms * g[e] : r[e] + v[e] / rms * g[e];
        reinterpret_cast<float4*>(x + base + c)[0] = make_float4(r[0], r[1], r[2], r[3]);
        reinterpret_cast<float4*>(x + base + c)[1] = make_float4(r[4], r[5], r[6], r[7]);
        if (xa) VecIO<__nv_bfloat16>::store(xa + base + c, r);
    };
    if constexpr (MAXV > 0) {
#pragma unroll
        for (int i = 0; i < MAXV; ++i) {
            const int c = (i * 256 + threadIdx.x) * 8;
            if (c < wp) update(c, keep[i], res[i]);
        }
    } else {
        for (int c = threadIdx.x * 8; c < wp; c += 2048) {
            float v[8], r[8];
            load8(y + base + c, v);
            load8(x + base + c, r);
            if (SUM)
#pragma unroll
                for (int e = 0; e < 8; ++e) v[e] = fmaf(alpha, r[e], v[e]);
            update(c, v, r);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(256) final_norm_kernel(const float* __restrict__ x, const int32_t* __restrict__ rows, const float* __restrict__ gain,
                                                         float eps, T* __restrict__ out, int d, int wp) {
    __shared__ float smem[8];
    constexpr int N = VecIO<T>::N;
    chain_trigger();
    chain_wait();
    const float* src = x + (long long)rows[blockIdx.x] * wp;
    float q = 0.0f;
    for (int c = threadIdx.x; c < d; c += 256) q = fmaf(src[c], src[c], q);
    q = block_sum(q, smem) / (float)d;
    const float rms = sqrtf(q + eps);
    for (int c = threadIdx.x * N; c < wp; c += 256 * N) {
        float v[N];
#pragma unroll
        for (int i = 0; i < N; ++i) v[i] = src[c + i] / rms * gain[c + i];
        VecIO<T>::store(out + (long long)blockIdx.x * wp + c, v);
    }
}

// Logits of one row per blockIdx.y, split over gridDim.x CTAs: the cap in place and the arg-max over the capped values.  A
// slice's best (value, index) becomes one monotone 64-bit key that goes into the row's key with atomicMax (larger value
// first, then the lower index); the CTA that arrives last writes the token and resets both words for the next launch.
__global__ void __launch_bounds__(256) logits_finish_kernel(float* __restrict__ logits, int pitch, int vocab, float cap,
                                                            unsigned long long* __restrict__ keys, int32_t* __restrict__ ctrs,
                                                            int32_t* __restrict__ next) {
    __shared__ unsigned long long best[8];
    chain_trigger();
    chain_wait();
    const int r = blockIdx.y;
    float* row = logits + (long long)r * pitch;
    const int lo = (int)((long long)blockIdx.x * vocab / gridDim.x), hi = (int)((long long)(blockIdx.x + 1) * vocab / gridDim.x);
    unsigned long long key = 0;  // below every value's key
    for (int i = lo + threadIdx.x; i < hi; i += 256) {
        float v = row[i];
        if (cap > 0.0f) {
            v = cap * tanhf(v / cap);
            row[i] = v;
        }
        const uint32_t bits = __float_as_uint(v);
        const uint32_t mono = (bits & 0x80000000u) ? ~bits : (bits | 0x80000000u);
        const unsigned long long k = ((unsigned long long)mono << 32) | (0xffffffffu - (uint32_t)i);
        if (v == v && k > key) key = k;
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const unsigned long long other = __shfl_xor_sync(0xffffffffu, key, o);
        if (other > key) key = other;
    }
    if ((threadIdx.x & 31) == 0) best[threadIdx.x >> 5] = key;
    __syncthreads();
    if (threadIdx.x == 0) {
#pragma unroll
        for (int w = 1; w < 8; ++w)
            if (best[w] > key) key = best[w];
        atomicMax(keys + r, key);
        __threadfence();
        if (atomicAdd(ctrs + r, 1) == (int)gridDim.x - 1) {
            __threadfence();
            const unsigned long long top = atomicExch(keys + r, 0ull);
            next[r] = top ? (int32_t)(0xffffffffu - (uint32_t)(top & 0xffffffffull)) : 0;
            ctrs[r] = 0;
        }
    }
}

__device__ __forceinline__ float clamped_glu(float g, float u, float alpha, float limit) {
    g = fminf(g, limit);
    u = fminf(fmaxf(u, -limit), limit);
    return g / (1.0f + expf(-alpha * g)) * (u + 1.0f);
}
__global__ void __launch_bounds__(256) clamped_glu_f32_kernel(const float* __restrict__ gate, const float* __restrict__ up, float* __restrict__ act,
                                                              float alpha, float limit, long long n) {
    chain_trigger();
    chain_wait();
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256)
        act[i] = clamped_glu(gate[i], up[i], alpha, limit);
}

jsm_status embed_residual_launch(bool f32, const void* table, const int32_t* ids, float scale, float* x, void* xa, int T, int wp, cudaStream_t st) {
    if (f32)
        JSM_CUDA_CHECK(launch_chained(embed_residual_kernel<float>, dim3(T), dim3(256), 0, st, (const float*)table, ids, x, (float*)nullptr, scale,
                                      wp));
    else
        JSM_CUDA_CHECK(launch_chained(embed_residual_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, st, (const __nv_bfloat16*)table, ids, x,
                                      (__nv_bfloat16*)xa, scale, wp));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

template <bool SUM>
static jsm_status norm_residual(const float* y, float* x, const float* gain, float eps, float alpha, void* xa, int T, int d, int wp, cudaStream_t st) {
    auto go = [&](auto kernel) { return launch_chained(kernel, dim3(T), dim3(256), 0, st, y, x, gain, eps, alpha, (__nv_bfloat16*)xa, d, wp); };
    JSM_CUDA_CHECK(wp <= 2048 ? go(post_norm_add_kernel<1, SUM>) : wp <= 4096 ? go(post_norm_add_kernel<2, SUM>) : go(post_norm_add_kernel<0, SUM>));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}
jsm_status post_norm_add_launch(const float* y, float* x, const float* gain, float eps, void* xa, int T, int d, int wp, cudaStream_t st) {
    return norm_residual<false>(y, x, gain, eps, 1.0f, xa, T, d, wp, st);
}
jsm_status sum_norm_launch(const float* y, float* x, const float* gain, float eps, float alpha, void* xa, int T, int d, int wp, cudaStream_t st) {
    return norm_residual<true>(y, x, gain, eps, alpha, xa, T, d, wp, st);
}

jsm_status final_norm_launch(bool f32, const float* x, const int32_t* rows, const float* gain, float eps, void* out, int n, int d, int wp,
                             cudaStream_t st) {
    if (n <= 0) return JSM_OK;
    if (f32)
        JSM_CUDA_CHECK(launch_chained(final_norm_kernel<float>, dim3(n), dim3(256), 0, st, x, rows, gain, eps, (float*)out, d, wp));
    else
        JSM_CUDA_CHECK(launch_chained(final_norm_kernel<__nv_bfloat16>, dim3(n), dim3(256), 0, st, x, rows, gain, eps, (__nv_bfloat16*)out, d, wp));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

jsm_status logits_finish_launch(float* logits, int pitch, int vocab, float cap, int rows, unsigned long long* keys, int32_t* ctrs, int32_t* next,
                                cudaStream_t st) {
    if (rows <= 0) return JSM_OK;
    const int slices = std::max(1, std::min(16, vocab / 1024));
    JSM_CUDA_CHECK(launch_chained(logits_finish_kernel, dim3(slices, rows), dim3(256), 0, st, logits, pitch, vocab, cap, keys, ctrs, next));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

__global__ void __launch_bounds__(256) gelu_glu_f32_kernel(const float* __restrict__ gate, const float* __restrict__ up, float* __restrict__ act, long long n) {
    chain_trigger();
    chain_wait();
    for (long long i = (long long)blockIdx.x * 256 + threadIdx.x; i < n; i += (long long)gridDim.x * 256) {
        const float z = gate[i];
        act[i] = 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z))) * up[i];
    }
}
jsm_status gelu_glu_f32_launch(const float* gate, const float* up, float* act, long long n, cudaStream_t st) {
    JSM_CUDA_CHECK(launch_chained(gelu_glu_f32_kernel, dim3((unsigned)std::min<long long>((n + 255) / 256, 148 * 16)), dim3(256), 0, st, gate, up, act, n));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

jsm_status clamped_glu_f32_launch(const float* gate, const float* up, float* act, float alpha, float limit, long long n, cudaStream_t st) {
    JSM_CUDA_CHECK(launch_chained(clamped_glu_f32_kernel, dim3((unsigned)std::min<long long>((n + 255) / 256, 148 * 16)), dim3(256), 0, st, gate, up, act,
                                  alpha, limit, n));
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

}  // namespace jsm

using namespace jsm;

extern "C" jsm_status jsm_embedding(const void* d_table, const void* d_pos_table, const int32_t* d_ids,
                                    const int32_t* d_positions, void* d_out, jsm_dtype dtype, int T, int d, void* stream) {
    if (T == 0) return JSM_OK;
    if (!d_table || !d_ids || !d_out) JSM_FAIL(JSM_INVALID_ARG, "jsm_embedding: null pointer");
    if (dtype == JSM_F32 && d % 4 == 0)
        JSM_CUDA_CHECK(launch_chained(embedding_kernel<float>, dim3(T), dim3(256), 0, as_stream(stream), (const float*)d_table,
                                      (const float*)d_pos_table, d_ids, d_positions, (float*)d_out, d));
    else if (dtype == JSM_BF16 && d % 8 == 0)
        JSM_CUDA_CHECK(launch_chained(embedding_kernel<__nv_bfloat16>, dim3(T), dim3(256), 0, as_stream(stream),
                                      (const __nv_bfloat16*)d_table, (const __nv_bfloat16*)d_pos_table, d_ids, d_positions,
                                      (__nv_bfloat16*)d_out, d));
    else
        JSM_FAIL(JSM_UNSUPPORTED, "jsm_embedding: dtype %d with d %d (d must be a multiple of 16 bytes)", (int)dtype, d);
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

extern "C" jsm_status jsm_add_norm(int kind, const void* d_h, const void* d_delta, void* d_h_out, void* d_y, jsm_dtype dtype,
                                   const float* d_gain, const float* d_bias, float eps, int T, int d, void* stream) {
    if (T == 0) return JSM_OK;
    if (!d_h || !d_y) JSM_FAIL(JSM_INVALID_ARG, "jsm_add_norm: null pointer");
    if (kind != JSM_ROWS_LAYERNORM && kind != JSM_ROWS_RMSNORM) JSM_FAIL(JSM_INVALID_ARG, "jsm_add_norm: kind %d", kind);
    cudaStream_t st = as_stream(stream);
    if (dtype == JSM_F32) {
        if (d % 4 || d > 256 * 4 * 4) JSM_FAIL(JSM_UNSUPPORTED, "jsm_add_norm: f32 needs d %% 4 == 0 and d <= 4096 (d %d)", d);
        add_norm_kernel<float, 4><<<T, 256, 0, st>>>(kind, (const float*)d_h, (const float*)d_delta, (float*)d_h_out,
                                                     (float*)d_y, d_gain, d_bias, eps, d);
    } else if (dtype == JSM_BF16) {
        if (d % 8 || d > 256 * 8 * 4) JSM_FAIL(JSM_UNSUPPORTED, "jsm_add_norm: bf16 needs d %% 8 == 0 and d <= 8192 (d %d)", d);
        if (d <= 256 * 8 * 2)
            add_norm_kernel<__nv_bfloat16, 2><<<T, 256, 0, st>>>(kind, (const __nv_bfloat16*)d_h, (const __nv_bfloat16*)d_delta,
                                                                (__nv_bfloat16*)d_h_out, (__nv_bfloat16*)d_y, d_gain, d_bias, eps, d);
        else
            add_norm_kernel<__nv_bfloat16, 4><<<T, 256, 0, st>>>(kind, (const __nv_bfloat16*)d_h, (const __nv_bfloat16*)d_delta,
                                                                (__nv_bfloat16*)d_h_out, (__nv_bfloat16*)d_y, d_gain, d_bias, eps, d);
    } else {
        JSM_FAIL(JSM_UNSUPPORTED, "jsm_add_norm: dtype %d", (int)dtype);
    }
    JSM_LAUNCH_CHECK();
    return JSM_OK;
}

extern "C" jsm_status jsm_post_norm_add(const float* d_y, float* d_x, const float* d_gain, float eps, void* d_x_bf16, int T, int d, void* stream) {
    if (T <= 0) return JSM_OK;
    if (!d_y || !d_x || !d_gain) JSM_FAIL(JSM_INVALID_ARG, "jsm_post_norm_add: null pointer");
    if (d <= 0 || d % 8) JSM_FAIL(JSM_UNSUPPORTED, "jsm_post_norm_add: d %d (a multiple of 8)", d);
    return post_norm_add_launch(d_y, d_x, d_gain, eps, d_x_bf16, T, d, d, as_stream(stream));
}

extern "C" jsm_status jsm_sum_norm(const float* d_y, float* d_x, const float* d_gain, float eps, float alpha, void* d_x_bf16, int T, int d, void* stream) {
    if (T <= 0) return JSM_OK;
    if (!d_y || !d_x || !d_gain) JSM_FAIL(JSM_INVALID_ARG, "jsm_sum_norm: null pointer");
    if (d <= 0 || d % 8) JSM_FAIL(JSM_UNSUPPORTED, "jsm_sum_norm: d %d (a multiple of 8)", d);
    return sum_norm_launch(d_y, d_x, d_gain, eps, alpha, d_x_bf16, T, d, d, as_stream(stream));
}

extern "C" jsm_status jsm_logits_finish(float* d_logits, int pitch, int rows, int vocab, float cap, uint64_t* d_keys, int32_t* d_counters,
                                        int32_t* d_next, void* stream) {
    if (rows <= 0) return JSM_OK;
    if (!d_logits || !d_keys || !d_counters || !d_next) JSM_FAIL(JSM_INVALID_ARG, "jsm_logits_finish: null pointer");
    if (vocab <= 0 || pitch < vocab) JSM_FAIL(JSM_SHAPE, "jsm_logits_finish: rows of %d logits, pitch %d", vocab, pitch);
    return logits_finish_launch(d_logits, pitch, vocab, cap, rows, reinterpret_cast<unsigned long long*>(d_keys), d_counters, d_next, as_stream(stream));
}
