// Internal interface of the mechanisms a layer-list decoder (decoder.cu) is composed of: latent attention over a paged
// latent cache, the selective scan with its short convolution, the norm on a sublayer's output, the capped logits.
// Activations are bf16 or f32 ("act" pointers, selected by the f32 flag); row pitches are multiples of 8 elements whose
// padding columns hold zeros.
#pragma once
#include "common.cuh"

namespace jsm {

int* tc_error_word();

__host__ __device__ inline int pad8(int n) { return (n + 7) & ~7; }
inline int pad_to(int n, int m) { return (n + m - 1) / m * m; }

// The tokens of one pass, grouped in segments: consecutive positions of one sequence each.  All arrays on the device.
struct StepTokens {
    int T = 0, n_segs = 0, max_len = 0;  // max_len: longest segment
    const int32_t* ids = nullptr;        // [T]
    const int32_t* tok_row = nullptr;    // [T] batch row (= row of the block table)
    const int32_t* tok_pos = nullptr;    // [T] position in its sequence
    const int32_t* seg_start = nullptr;  // [n_segs] first token
    const int32_t* seg_len = nullptr;
    const int32_t* seg_pos0 = nullptr;   // position of the first token
    const int32_t* seg_row = nullptr;
    const int32_t* seg_slot = nullptr;   // recurrent-state slot of the sequence
};

// ---- latent attention (latent_attn.cu) ----------------------------------------------------------------------------
// Per head: `dim` unrotated and `rot` rotated query / key components, values of `vdim`.  Keys and values are linear in a
// latent c of `rank` components, so a token's cache entry is [c | rotated key part], rank + rot components (pitch cr).
struct LatentDims {
    int H, dim, rot, vdim, rank, window;
    float scale;
    int qh() const { return pad8(dim + rot); }        // pitch of one head's query
    int cr() const { return pad8(rank + rot); }       // pitch of a cache entry
    int q_cols() const { return H * qh(); }
    int down_cols() const { return pad8(rank + rot); }
    int out_cols() const { return pad8(H * vdim); }
    int dkp() const { return pad_to(dim + rot, 64); } // expanded key / value pitches per head (tensor-core tiles)
    int dvp() const { return pad_to(vdim, 64); }
};
struct LatentWeights {
    const float* down_norm;  // gain of the latent's RMS norm, [rank]
    const void* uk;          // act dtype, per head transposed: [H][nk][kk], nk = pad(rank, 16), kk = pad(dim, 32)
    const void* uv;          // [H][nv][kv], nv = pad(vdim, 16), kv = pad(rank, 32)
};
struct LatentCache {
    void* pool;              // act dtype, [pages][64][cr]
    const int32_t* block_table;
    int max_pages;
    const float2* rope;      // (cos, sin) of [position][rot / 2]
};
// From the fused down/query projection qd (f32 [T][q_cols + down_cols]): appends [norm(c) | rotated key part] to the
// cache and writes the queries, rotated, to q (act [T][q_cols]); the rotated parts also go into the latent queries q_lat
// (act [T][H][cr], behind their rank columns; may be null).
jsm_status latent_prep_launch(bool f32, const float* qd, const LatentDims& d, const LatentWeights& w, float eps, const LatentCache& cache,
                              const StepTokens& tk, void* q, void* q_lat, cudaStream_t st);
// Attention in the latent space for the tokens listed in tiles: queries are taken into the latent space (the rank columns of q_lat), scored
// against the cache, and the weighted latents (o_lat) expanded to values: out act [T][out_cols].
struct LatentScratch {
    void* q_lat;             // act [T][H][cr]
    void* o_lat;             // act [T][H][pad8(rank)]
    float* part;             // split partials
    size_t part_floats;
};
constexpr int LATENT_TILE_ROWS = 32;  // (token, head) rows per CTA of the tensor-core kernel
// tiles: tile_seg / tile_r0 (device), rows r0 .. r0+31 of segment tile_seg in (token, head) order.  t_first / t_count: the
// token range the query / output expansions run over (covers the tiles' tokens).
struct LatentTiles { const int32_t* tile_seg; const int32_t* tile_r0; int n_tiles; int t_first, t_count; int max_keys; };
bool latent_mma_usable(const LatentDims& d);
int latent_splits(int n_tiles, int max_keys);
size_t latent_part_floats(const LatentDims& d);
jsm_status latent_attn_launch(bool f32, const LatentDims& d, const LatentWeights& w, const LatentCache& cache, const StepTokens& tk,
                              const LatentTiles& tiles, const void* q, const LatentScratch& sc, void* out, cudaStream_t st);
// Long segments: keys and values expanded once per key (k [n_keys][H dkp], v [n_keys][H dvp] at pitch kv_pitch), then the
// flash kernel over a sliding window; the segment's queries are the last n_q of the n_keys positions.
bool latent_flash_usable(const LatentDims& d);
jsm_status latent_flash_launch(const LatentDims& d, const void* q, const void* k, const void* v, long long kv_pitch, void* out, int n_q, int n_keys,
                               cudaStream_t st);
// Contiguous copy of the cache entries of positions [p0, p0 + n) of batch row `row`: bf16 [n][cr]
jsm_status latent_gather_launch(const LatentDims& d, const LatentCache& cache, int row, int p0, int n, void* out, cudaStream_t st);

// ---- grouped-query attention over a paged cache (paged_attn.cu) -----------------------------------------------------
// Keys a query sees: all before it, the last `size`, or those of its own chunk of `size` positions (counted from 0).
struct KeyMask {
    int kind = JSM_MASK_FULL, size = 0;
    __host__ __device__ int first(int pos) const {
        return kind == JSM_MASK_CHUNK ? pos - pos % size : kind == JSM_MASK_WINDOW && pos >= size ? pos - size + 1 : 0;
    }
    int reach(int max_context) const { return kind == JSM_MASK_FULL || size > max_context ? max_context : size; }  // most keys of a query
};
struct AttnDims {
    int H = 0, G = 0, dim = 0, vdim = 0, rot = 0;
    KeyMask mask;
    float scale = 0.0f;
    int gated = 0;                                                        // a gate per head on the output
    __host__ __device__ int qh() const { return pad8(dim); }              // pitch of one head's query / key in a row
    __host__ __device__ int ks() const { return (dim + 63) / 64; }        // 64-column slabs of a key / value in the cache
    __host__ __device__ int vs() const { return (vdim + 63) / 64; }
    __host__ __device__ int q_cols() const { return H * qh(); }
    __host__ __device__ int out_cols() const { return pad8(H * vdim); }
    __host__ __device__ int wide_cols(bool kv) const { return q_cols() + pad8(H) + (kv ? G * (qh() + pad8(vdim)) : 0); }  // [q | gates | k | v]
    size_t page_elems() const { return (size_t)G * (ks() + vs()) * JSM_PAGE_SIZE * 64; }
};
struct AttnWeights {  // f32; null: the design has none.  Biases at the pitches of the projection, norms [dim], sink [H]
    const float *q_bias = nullptr, *k_bias = nullptr, *v_bias = nullptr, *q_norm = nullptr, *k_norm = nullptr, *sink = nullptr;
};
struct AttnCache {
    void* pool = nullptr;  // act dtype, [pages][G][ks + vs][64][64], swizzled
    const int32_t* block_table = nullptr;
    int max_pages = 0;
    const float2* rope = nullptr;  // (cos, sin) of [position][rot / 2]
};
// From the fused projection wide (f32 [T][wide_cols]): queries (act [T][q_cols]), gates (f32 [T][H], after the sigmoid), and
// the cache entries of the pass's tokens (own_kv)
jsm_status attn_prep_launch(bool f32, const float* wide, const AttnDims& d, const AttnWeights& w, float eps, const AttnCache& cache, bool own_kv,
                            const StepTokens& tk, void* q, float* gate, cudaStream_t st);
struct AttnScratch { float* part; size_t part_floats; int* counters; int n_counters; };  // counters: zero before the first launch
// tiles: rows r0 .. r0 + rows - 1 of segment tile_seg in (token, head of the group) order
struct AttnTiles { const int32_t* tile_seg; const int32_t* tile_r0; int n_tiles, rows, t_first, t_count, max_keys; };
bool attn_mma_usable(const AttnDims& d);
int attn_tile_rows(const AttnDims& d, bool decode);
size_t attn_part_floats(const AttnDims& d);
int attn_counters();
jsm_status attn_paged_launch(bool f32, const AttnDims& d, const AttnWeights& w, const AttnCache& cache, const StepTokens& tk, const AttnTiles& tiles,
                             const void* q, const float* gate, const AttnScratch& sc, void* out, cudaStream_t st);
// Long segments on the flash kernel, straight from the pages (flash_attn.cu); q and out: the segment's first row
bool attn_flash_usable(const AttnDims& d);
jsm_status attn_flash_launch(const AttnDims& d, const AttnWeights& w, const AttnCache& cache, int row, int pos0, int len, const void* q, const float* gate,
                             void* out, cudaStream_t st);

// ---- selective scan (selective_scan.cu) ---------------------------------------------------------------------------
struct ScanDims {
    int inner, state, dt_rank, taps;
    int ip() const { return pad8(inner); }
    int np() const { return pad8(state); }
    int rp() const { return pad8(dt_rank); }
    int proj_cols() const { return rp() + 2 * np(); }  // [dt | B | C]
};
struct ScanWeights {
    const float *conv, *conv_b;  // [taps][ip], [ip]
    const float* A;              // [np / 4][ip][4]: -exp(A_log) (0 in the padding)
    const float* D;              // [ip]
    const float* dt_b;           // [ip]
    const void* dt;              // act dtype, [ip][rp] (the fused decode step)
};
struct ScanState {
    void* conv;    // act [slots][taps - 1][ip]: the last inputs of the convolution
    float* S;      // [slots][np / 4][ip][4]
};
// xc = silu(conv(x) + b) over the x half of xz (act [T][2 ip]); carry (one token per segment): also moves the convolution
// state on, which otherwise the scan does
jsm_status scan_conv_launch(bool f32, const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz,
                            void* xc, bool carry, cudaStream_t st);
// the scan over every segment: proj f32 [T][proj_cols], dt_raw f32 [T][ip] (before bias and softplus); y act [T][ip] is
// gated by silu(z); carries the recurrent and the convolution state
jsm_status scan_launch(bool f32, const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz,
                       const void* xc, const float* proj, const float* dt_raw, void* y, cudaStream_t st);
// the same for one token per segment, with the step-size projection fused in
jsm_status scan_step_launch(bool f32, const ScanDims& d, const ScanWeights& w, const ScanState& s, const StepTokens& tk, const void* xz,
                            const void* xc, const float* proj, void* y, cudaStream_t st);
// the dt columns of proj as a bf16 operand [T][rp]
jsm_status scan_dt_operand_launch(const ScanDims& d, const float* proj, void* out, int T, cudaStream_t st);

// ---- short causal convolution (selective_scan.cu) -----------------------------------------------------------------
// out = silu(conv(x) + bias) over `cp` channels (a multiple of 8): x act [T][x_pitch], out act [T][cp], w f32 [taps][cp], bias
// f32 [cp] or null; state act [slots][taps - 1][cp]: the last inputs.  carry (one token per segment): also moves the state
// on; otherwise short_conv_carry_launch does that, after the convolution.
jsm_status short_conv_launch(bool f32, const void* x, long long x_pitch, int cp, int taps, const float* w, const float* bias, void* state,
                             const StepTokens& tk, void* out, bool carry, cudaStream_t st);
jsm_status short_conv_carry_launch(bool f32, const void* x, long long x_pitch, int cp, int taps, void* state, const StepTokens& tk, cudaStream_t st);

// ---- linear recurrences with a matrix state (linear_recurrence.cu) ------------------------------------------------
struct RecDims {
    int H = 0, G = 0, dk = 0, dv = 0, taps = 0;
    bool delta = false;                                                              // delta rule, or a decayed sum
    __host__ __device__ int kp() const { return pad8(dk); }
    __host__ __device__ int vp() const { return pad8(dv); }
    __host__ __device__ int conv_cols() const { return 2 * G * kp() + H * vp(); }    // [q | k | v]
    __host__ __device__ int raw_cols() const { return conv_cols() + H * vp(); }      // [q | k | v | z]
    __host__ __device__ int ba_cols() const { return delta ? 2 * pad8(H) : 0; }      // [b | a]
    int out_cols() const { return H * vp(); }
};
struct RecWeights {
    const float* conv = nullptr;                              // [taps][conv cols]
    const float *A = nullptr, *dt_bias = nullptr;             // [H]: -exp(A_log); delta rule
    const float *decay = nullptr, *log_decay = nullptr;       // [H]; decayed sum
    const float* norm = nullptr;                              // [vp] (delta rule) or [H vp]
    const void* ba = nullptr;                                 // act [ba cols][x pitch] (the fused decode step)
};
struct RecState {
    void* conv = nullptr;  // act [slots][taps - 1][conv cols]
    float* S = nullptr;    // [slots][H][kp][vp]
};
constexpr int REC_CHUNK = 64;  // tokens of a chunk of the tensor-core kernels
// The chunks of a pass: segment by segment, the last one of a segment may be short.  ws: rec_chunk_bytes per chunk.
struct RecChunks {
    const int32_t *chunk_seg = nullptr, *chunk_t0 = nullptr;  // [n_chunks] segment, first token within it
    const int32_t* seg_chunk0 = nullptr;                      // [n_segs] first chunk
    int n_chunks = 0;
    void* ws = nullptr;
};
bool rec_usable(const RecDims& d);
bool rec_chunk_usable(const RecDims& d);
size_t rec_chunk_bytes(const RecDims& d);
// raw: the input projection; qkv: its first columns after the convolution; ba f32 [T][ba cols]; out act [T][H vp]: normed, gated
jsm_status rec_scan_launch(bool f32, const RecDims& d, const RecWeights& w, const RecState& s, float eps, const StepTokens& tk, const RecChunks& ch,
                           const void* raw, const void* qkv, const float* ba, void* out, cudaStream_t st);
// the same for one token per segment; b and a come from the layer's input x (act [T][x_pitch])
jsm_status rec_step_launch(bool f32, const RecDims& d, const RecWeights& w, const RecState& s, float eps, const StepTokens& tk, const void* raw,
                           const void* qkv, const void* x, int x_pitch, void* out, cudaStream_t st);

// ---- token-level (tokens.cu) --------------------------------------------------------------------------------------
// x[t] = table[ids[t]] * scale in f32, and its bf16 copy xa (or null); table act [vocab][wp]
jsm_status embed_residual_launch(bool f32, const void* table, const int32_t* ids, float scale, float* x, void* xa, int T, int wp, cudaStream_t st);
// x += y / rms(y) * gain over the first d of wp columns; xa (bf16 copy, or null)
jsm_status post_norm_add_launch(const float* y, float* x, const float* gain, float eps, void* xa, int T, int d, int wp, cudaStream_t st);
// x <- s / rms(s) * gain, s = alpha x + y
jsm_status sum_norm_launch(const float* y, float* x, const float* gain, float eps, float alpha, void* xa, int T, int d, int wp, cudaStream_t st);
// out[i] = x[rows[i]] / rms * gain, act [n][wp]
jsm_status final_norm_launch(bool f32, const float* x, const int32_t* rows, const float* gain, float eps, void* out, int n, int d, int wp,
                             cudaStream_t st);
// logits <- cap * tanh(logits / cap) in place (cap <= 0: unchanged) and the arg-max of every row (first maximum)
jsm_status logits_finish_launch(float* logits, int pitch, int vocab, float cap, int rows, unsigned long long* keys, int32_t* ctrs,
                                int32_t* next, cudaStream_t st);
// act = min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u, -limit, limit) + 1), all f32 [T][n]
jsm_status clamped_glu_f32_launch(const float* gate, const float* up, float* act, float alpha, float limit, long long n, cudaStream_t st);
// act = gelu_tanh(gate) * up, all f32
jsm_status gelu_glu_f32_launch(const float* gate, const float* up, float* act, long long n, cudaStream_t st);

}  // namespace jsm
