// Internal interface of the mechanisms a layer-list decoder (decoder.cu) is composed of: latent attention over a paged
// latent cache, the selective scan with its short convolution, the norm on a sublayer's output, the capped logits.
// Activations are bf16 or f32 ("act" pointers, selected by the f32 flag); row pitches are multiples of 8 elements whose
// padding columns hold zeros.
#pragma once
#include "common.cuh"

namespace jsm {

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

// ---- token-level (tokens.cu) --------------------------------------------------------------------------------------
// x[t] = table[ids[t]] in f32, and its bf16 copy xa (or null); table act [vocab][wp]
jsm_status embed_residual_launch(bool f32, const void* table, const int32_t* ids, float* x, void* xa, int T, int wp, cudaStream_t st);
// x += y / rms(y) * gain over the first d of wp columns; xa (bf16 copy, or null)
jsm_status post_norm_add_launch(const float* y, float* x, const float* gain, float eps, void* xa, int T, int d, int wp, cudaStream_t st);
// out[i] = x[rows[i]] / rms * gain, act [n][wp]
jsm_status final_norm_launch(bool f32, const float* x, const int32_t* rows, const float* gain, float eps, void* out, int n, int d, int wp,
                             cudaStream_t st);
// logits <- cap * tanh(logits / cap) in place (cap <= 0: unchanged) and the arg-max of every row (first maximum)
jsm_status logits_finish_launch(float* logits, int pitch, int vocab, float cap, int rows, unsigned long long* keys, int32_t* ctrs,
                                int32_t* next, cudaStream_t st);
// act = min(g, limit) * sigmoid(alpha * min(g, limit)) * (clamp(u, -limit, limit) + 1), all f32 [T][n]
jsm_status clamped_glu_f32_launch(const float* gate, const float* up, float* act, float alpha, float limit, long long n, cudaStream_t st);

}  // namespace jsm
