// Decoder whose layers are a list: every layer names its mixer (latent attention, grouped-query attention, a selective scan, a
// decayed sum or the delta rule), the mixer's sizes, and an optional gated feed-forward.  The norm sits on the sublayer's output,
//     x <- x + norm1(mixer(x)),   x <- x + norm2(ff(x)),
// or on the sum, x <- norm1(alpha x + mixer(x)); the residual stream x is fp32, the logits come from the embedding table and
// may pass through a soft cap.  A layer may use the weights of an earlier one with a cache or state of its own, and an
// attention layer the keys and values of an earlier one.
//
// Serving follows the paged LLaMA runner (llama.cu, paged_rows.cuh): the active sequences occupy the batch rows
// 0 .. n_active-1, cache pages of 64 positions come from one pool (all attention layers share the block table),
// pages that no mask reaches any more go back to the pool, and every sequence owns one recurrent-state slot.  One step
// function runs everything: a step brings tokens of any number of rows - a prompt, a portion of one, one token each - and
// is cut into passes of at most max_step_tokens.  A pass whose rows bring one token each replays a CUDA graph.
//
// bf16: weights packed for the tensor-core projections, activations bf16, residual, norms, scores, recurrences and logits
// fp32.  f32: fp32 weights, activations and products throughout (dot_f32.cu and the f32 forms of the kernels).
#include "common.cuh"
#include "decoder_ops.cuh"
#include "linear_bf16.cuh"
#include "attn.cuh"
#include "paged_rows.cuh"
#include <math.h>
#include <string.h>
#include <algorithm>
#include <map>
#include <string>
#include <vector>

namespace jsm {

int* tc_error_word();
jsm_status dot_f32_launch(const jsm_mat& A, const jsm_mat& B, const jsm_mat& C, cudaStream_t st);

struct Proj {  // one projection: N outputs, K inputs, both rounded up to multiples of 8 (zero rows / columns)
    int N = 0, K = 0, paired = 0;
    uint8_t* packed = nullptr;  // bf16 models
    float* w32 = nullptr;       // f32 models, [N][K]
    void* rows = nullptr;       // bf16 models, projections with few outputs or few inputs: also row-major, for many tokens
};

struct DecLayer {
    jsm_layer_config c;
    LatentDims ld{};
    ScanDims sd{};
    AttnDims ad{};
    RecDims rd{};
    const float *norm1 = nullptr, *norm2 = nullptr;
    Proj qd, expand, in, xp, dt, out;  // latent: queries + down projection, key / value expansion; scan: input, [dt B C], dt; all: output
                                       // attention: qd = [q | gates | k | v]; recurrences: in = [q | k | v | z], xp = [b | a]
    Proj gate, up, down;               // bf16: gate holds the gate / up pairs
    LatentWeights lw{};
    ScanWeights sw{};
    LatentCache cache{};
    ScanState state{};
    AttnWeights aw{};
    AttnCache ac{};
    RecWeights rw{};
    RecState rs{};
    bool is_attention() const { return c.mixer == JSM_MIXER_LATENT_ATTENTION || c.mixer == JSM_MIXER_ATTENTION; }
    bool is_recurrence() const { return c.mixer == JSM_MIXER_LINEAR_ATTENTION || c.mixer == JSM_MIXER_DELTA; }
    bool own_kv() const { return c.kv_from < 0; }
    // rows per token and rows per tile of the tensor-core attention kernels
    std::pair<int, int> tiling(bool decode) const {
        return c.mixer == JSM_MIXER_LATENT_ATTENTION ? std::make_pair(ld.H, LATENT_TILE_ROWS) : std::make_pair(ad.H / ad.G, attn_tile_rows(ad, decode));
    }
    KeyMask key_mask() const { return c.mixer == JSM_MIXER_LATENT_ATTENTION ? KeyMask{JSM_MASK_WINDOW, c.window} : ad.mask; }
    int ffp() const { return pad8(c.ff); }
};

struct HostTensor {
    int rows = 0, cols = 0;
    std::vector<float> v;
    std::vector<uint16_t> b;  // one of the two
    float at(long long i) const { return v.empty() ? bf16_bits_to_f32(b[i]) : v[i]; }
};

struct PassSeg { int entry, row, tok0, len, pos0; };  // tok0: first token within the step's flat token list

constexpr float GLU_ALPHA = 1.702f;   // slope of the gate's sigmoid
constexpr int FLASH_MIN_TOKENS = 128; // segments from this length on expand keys and values and run the flash kernel

}  // namespace jsm

struct jsm_decoder {
    jsm_decoder_config c;
    bool f32 = false, ready = false;
    std::vector<jsm::DecLayer> layers;
    std::map<std::string, jsm::HostTensor> tensors;  // until jsm_decoder_finalize
    void* embed = nullptr;                           // act [vocab][wp]
    jsm::Proj head;
    const float* final_norm = nullptr;
    jsm::PagedRows rows;
    std::vector<int> slot_of_row, free_slots;
    int wp = 0, vp = 0, cap_rows = 0, kv_rows = 0;
    bool has_attention = false;
    cudaStream_t own_stream = nullptr;
    std::vector<void*> allocs;
    // activations of one pass
    float *x = nullptr, *y = nullptr, *wide = nullptr, *proj = nullptr, *dt_raw = nullptr, *gate32 = nullptr, *head_gate = nullptr, *logits = nullptr, *part = nullptr;
    void *xa = nullptr, *q = nullptr, *q_lat = nullptr, *o_lat = nullptr, *att = nullptr, *xz = nullptr, *xc = nullptr, *dt_op = nullptr,
         *scan_y = nullptr, *act = nullptr, *head_in = nullptr, *gathered = nullptr, *expanded = nullptr;
    size_t part_floats = 0, chunk_bytes = 0;
    void* chunk_ws = nullptr;
    float* ws = nullptr;
    size_t ws_floats = 0;
    int* counters = nullptr;
    int n_counters = 0;
    int* attn_ctrs = nullptr;
    unsigned long long* keys = nullptr;
    int32_t *key_ctrs = nullptr, *next_dev = nullptr, *meta = nullptr, *h_meta = nullptr;
    size_t meta_cap = 0;
    std::map<int, cudaGraphExec_t> graphs;
    float* tap = nullptr;
    uint64_t weight_bytes = 0;
};

namespace jsm {

template <typename T>
static jsm_status dalloc(jsm_decoder* m, T** p, size_t bytes) {
    void* q = nullptr;
    if (bytes == 0) bytes = 16;
    cudaError_t e = cudaMalloc(&q, bytes);
    if (e == cudaSuccess) {
        m->allocs.push_back(q);
        e = cudaMemset(q, 0, bytes);
    }
    if (e != cudaSuccess) {
        cudaGetLastError();
        JSM_FAIL(JSM_OOM, "jsm_decoder: allocation of %zu bytes failed: %s", bytes, cudaGetErrorString(e));
    }
    *p = reinterpret_cast<T*>(q);
    return JSM_OK;
}

// A zero-initialised host matrix in the model's weight type
struct HostMatrix {
    bool f32;
    int N, K;
    std::vector<float> v;
    std::vector<uint16_t> b;
    HostMatrix(bool f32_, int N_, int K_) : f32(f32_), N(N_), K(K_) {
        if (f32) v.assign((size_t)N * K, 0.0f);
        else b.assign((size_t)N * K, 0);
    }
    void set(int r, int c, float x) {
        if (f32) v[(size_t)r * K + c] = x;
        else b[(size_t)r * K + c] = f32_to_bf16_bits(x);
    }
    void put_row(int r, const HostTensor& t, int tr) {
        if (!f32 && t.v.empty()) memcpy(&b[(size_t)r * K], &t.b[(size_t)tr * t.cols], sizeof(uint16_t) * t.cols);
        else
            for (int c = 0; c < t.cols; ++c) set(r, c, t.at((long long)tr * t.cols + c));
    }
    size_t bytes() const { return f32 ? v.size() * 4 : b.size() * 2; }
    const void* data() const { return f32 ? (const void*)v.data() : (const void*)b.data(); }
};

static jsm_status upload_plain(jsm_decoder* m, const HostMatrix& h, void** out) {
    jsm_status s = dalloc(m, out, h.bytes());
    if (s != JSM_OK) return s;
    JSM_CUDA_CHECK(cudaMemcpy(*out, h.data(), h.bytes(), cudaMemcpyHostToDevice));
    return JSM_OK;
}
// paired: h holds the gate rows, then the up rows
static jsm_status upload_proj(jsm_decoder* m, const HostMatrix& h, Proj* p, bool paired = false) {
    p->N = paired ? h.N / 2 : h.N;
    p->K = h.K;
    p->paired = paired ? 1 : 0;
    if (m->f32) return upload_plain(m, h, reinterpret_cast<void**>(&p->w32));
    jsm_status s = dalloc(m, &p->packed, linear_packed_bytes(p->N, p->K, p->paired));
    if (s != JSM_OK) return s;
    void* tmp = nullptr;
    JSM_CUDA_CHECK(cudaMalloc(&tmp, h.bytes()));
    cudaError_t e = cudaMemcpy(tmp, h.data(), h.bytes(), cudaMemcpyHostToDevice);
    if (e == cudaSuccess) {
        s = linear_pack_launch(tmp, p->N, p->K, p->paired, p->packed, false, nullptr);
        e = cudaDeviceSynchronize();
    }
    cudaFree(tmp);
    if (s != JSM_OK) return s;
    JSM_CUDA_CHECK(e);
    m->ws_floats = std::max(m->ws_floats, linear_packed_ws_floats(256, p->N, p->K, p->paired));
    m->n_counters = std::max(m->n_counters, (p->paired ? (p->N + 63) / 64 : (p->N + 127) / 128) + 1);
    return JSM_OK;
}
static jsm_status upload_vec(jsm_decoder* m, const HostTensor& t, int n_pad, const float** out) {
    std::vector<float> v(n_pad, 0.0f);
    for (int i = 0; i < t.rows * t.cols; ++i) v[i] = t.at(i);
    float* d = nullptr;
    jsm_status s = dalloc(m, &d, sizeof(float) * n_pad);
    if (s != JSM_OK) return s;
    JSM_CUDA_CHECK(cudaMemcpy(d, v.data(), sizeof(float) * n_pad, cudaMemcpyHostToDevice));
    *out = d;
    return JSM_OK;
}

static jsm_status want_tensor(jsm_decoder* m, const std::string& name, int rows, int cols, const HostTensor** out) {
    auto it = m->tensors.find(name);
    if (it == m->tensors.end()) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder: tensor '%s' is missing", name.c_str());
    if (it->second.rows != rows || it->second.cols != cols)
        JSM_FAIL(JSM_SHAPE, "jsm_decoder: tensor '%s' is [%d, %d], the configuration needs [%d, %d]", name.c_str(), it->second.rows,
                 it->second.cols, rows, cols);
    *out = &it->second;
    return JSM_OK;
}

#define DEC_TRY(x)                       \
    do {                                 \
        jsm_status s__ = (x);            \
        if (s__ != JSM_OK) return s__;   \
    } while (0)

static jsm_status build_latent(jsm_decoder* m, DecLayer& L, const std::string& pre) {
    const LatentDims& d = L.ld;
    const int D = m->c.d_model, wp = m->wp;
    const HostTensor *q, *dkv, *nrm, *uk, *uv, *o;
    DEC_TRY(want_tensor(m, pre + "mix.q", d.H * (d.dim + d.rot), D, &q));
    DEC_TRY(want_tensor(m, pre + "mix.dkv", d.rank + d.rot, D, &dkv));
    DEC_TRY(want_tensor(m, pre + "mix.dkv.norm", d.rank, 1, &nrm));
    DEC_TRY(want_tensor(m, pre + "mix.uk", d.H * d.dim, d.rank, &uk));
    DEC_TRY(want_tensor(m, pre + "mix.uv", d.H * d.vdim, d.rank, &uv));
    DEC_TRY(want_tensor(m, pre + "mix.o", D, d.H * d.vdim, &o));
    {
        HostMatrix h(m->f32, d.q_cols() + d.down_cols(), wp);
        for (int hd = 0; hd < d.H; ++hd)
            for (int j = 0; j < d.dim + d.rot; ++j) h.put_row(hd * d.qh() + j, *q, hd * (d.dim + d.rot) + j);
        for (int j = 0; j < d.rank + d.rot; ++j) h.put_row(d.q_cols() + j, *dkv, j);
        DEC_TRY(upload_proj(m, h, &L.qd));
    }
    {
        HostMatrix h(m->f32, wp, d.out_cols());
        for (int j = 0; j < D; ++j) h.put_row(j, *o, j);
        DEC_TRY(upload_proj(m, h, &L.out));
    }
    DEC_TRY(upload_vec(m, *nrm, pad8(d.rank), &L.lw.down_norm));
    {
        const int nk = pad_to(d.rank, 16), kk = pad_to(d.dim, 32);
        HostMatrix h(m->f32, d.H * nk, kk);
        for (int hd = 0; hd < d.H; ++hd)
            for (int j = 0; j < d.dim; ++j)
                for (int r = 0; r < d.rank; ++r) h.set(hd * nk + r, j, uk->at((long long)(hd * d.dim + j) * d.rank + r));
        void* p = nullptr;
        DEC_TRY(upload_plain(m, h, &p));
        L.lw.uk = p;
    }
    {
        const int nv = pad_to(d.vdim, 16), kv = pad_to(d.rank, 32);
        HostMatrix h(m->f32, d.H * nv, kv);
        for (int hd = 0; hd < d.H; ++hd)
            for (int j = 0; j < d.vdim; ++j) h.put_row(hd * nv + j, *uv, hd * d.vdim + j);
        void* p = nullptr;
        DEC_TRY(upload_plain(m, h, &p));
        L.lw.uv = p;
    }
    if (!m->f32 && latent_flash_usable(d)) {
        // one matrix takes a cache entry [c | rotated key part] to every head's key (an identity block passes the rotated
        // part through) and value, padded to the tiles of the flash kernel
        HostMatrix h(false, d.H * (d.dkp() + d.dvp()), d.cr());
        for (int hd = 0; hd < d.H; ++hd) {
            for (int j = 0; j < d.dim; ++j) h.put_row(hd * d.dkp() + j, *uk, hd * d.dim + j);
            for (int j = 0; j < d.rot; ++j) h.set(hd * d.dkp() + d.dim + j, d.rank + j, 1.0f);
            for (int j = 0; j < d.vdim; ++j) h.put_row(d.H * d.dkp() + hd * d.dvp() + j, *uv, hd * d.vdim + j);
        }
        DEC_TRY(upload_proj(m, h, &L.expand));
    }
    return JSM_OK;
}

static jsm_status build_scan(jsm_decoder* m, DecLayer& L, const std::string& pre) {
    const ScanDims& d = L.sd;
    const int D = m->c.d_model, wp = m->wp, ip = d.ip();
    const HostTensor *in, *conv, *conv_b, *xp, *dt, *dt_b, *A, *Dv, *o;
    DEC_TRY(want_tensor(m, pre + "mix.in", 2 * d.inner, D, &in));
    DEC_TRY(want_tensor(m, pre + "mix.conv", d.inner, d.taps, &conv));
    DEC_TRY(want_tensor(m, pre + "mix.conv.b", d.inner, 1, &conv_b));
    DEC_TRY(want_tensor(m, pre + "mix.x", d.dt_rank + 2 * d.state, d.inner, &xp));
    DEC_TRY(want_tensor(m, pre + "mix.dt", d.inner, d.dt_rank, &dt));
    DEC_TRY(want_tensor(m, pre + "mix.dt.b", d.inner, 1, &dt_b));
    DEC_TRY(want_tensor(m, pre + "mix.A_log", d.inner, d.state, &A));
    DEC_TRY(want_tensor(m, pre + "mix.D", d.inner, 1, &Dv));
    DEC_TRY(want_tensor(m, pre + "mix.o", D, d.inner, &o));
    {
        HostMatrix h(m->f32, 2 * ip, wp);
        for (int j = 0; j < d.inner; ++j) {
            h.put_row(j, *in, j);
            h.put_row(ip + j, *in, d.inner + j);
        }
        DEC_TRY(upload_proj(m, h, &L.in));
    }
    {
        HostMatrix h(m->f32, d.proj_cols(), ip);
        for (int j = 0; j < d.dt_rank; ++j) h.put_row(j, *xp, j);
        for (int j = 0; j < d.state; ++j) {
            h.put_row(d.rp() + j, *xp, d.dt_rank + j);
            h.put_row(d.rp() + d.np() + j, *xp, d.dt_rank + d.state + j);
        }
        DEC_TRY(upload_proj(m, h, &L.xp));
        if (!m->f32) DEC_TRY(upload_plain(m, h, &L.xp.rows));
    }
    {
        HostMatrix h(m->f32, ip, d.rp());
        for (int j = 0; j < d.inner; ++j) h.put_row(j, *dt, j);
        DEC_TRY(upload_proj(m, h, &L.dt));
        if (!m->f32) DEC_TRY(upload_plain(m, h, &L.dt.rows));
        L.sw.dt = m->f32 ? (void*)L.dt.w32 : L.dt.rows;
    }
    {
        HostMatrix h(m->f32, wp, ip);
        for (int j = 0; j < D; ++j) h.put_row(j, *o, j);
        DEC_TRY(upload_proj(m, h, &L.out));
    }
    {
        HostMatrix c(true, d.taps, ip), a(true, d.np() / 4, ip * 4);
        for (int j = 0; j < d.inner; ++j) {
            for (int k = 0; k < d.taps; ++k) c.set(k, j, conv->at((long long)j * d.taps + k));
            for (int n = 0; n < d.state; ++n) a.set(n / 4, j * 4 + n % 4, (float)-exp((double)A->at((long long)j * d.state + n)));
        }
        void *pc = nullptr, *pa = nullptr;
        DEC_TRY(upload_plain(m, c, &pc));
        DEC_TRY(upload_plain(m, a, &pa));
        L.sw.conv = static_cast<float*>(pc);
        L.sw.A = static_cast<float*>(pa);
    }
    DEC_TRY(upload_vec(m, *conv_b, ip, &L.sw.conv_b));
    DEC_TRY(upload_vec(m, *dt_b, ip, &L.sw.dt_b));
    DEC_TRY(upload_vec(m, *Dv, ip, &L.sw.D));
    return JSM_OK;
}

// rows [n heads x dim] of a tensor at a pitch of `pitch` rows per head, from row r0 on
static void put_heads(HostMatrix& h, int r0, const HostTensor& t, int n, int dim, int pitch) {
    for (int i = 0; i < n; ++i)
        for (int j = 0; j < dim; ++j) h.put_row(r0 + i * pitch + j, t, i * dim + j);
}
// a vector [n heads x dim] (or a column of a matrix) at a pitch per head
static jsm_status upload_heads(jsm_decoder* m, const HostTensor& t, int n, int dim, int pitch, const float** out) {
    HostTensor p;
    p.rows = n * pitch; p.cols = 1;
    p.v.assign((size_t)n * pitch, 0.0f);
    for (int i = 0; i < n; ++i)
        for (int j = 0; j < dim; ++j) p.v[(size_t)i * pitch + j] = t.at((long long)i * dim + j);
    return upload_vec(m, p, pad8(n * pitch), out);
}

static jsm_status build_attention(jsm_decoder* m, DecLayer& L, const std::string& pre) {
    const AttnDims& d = L.ad;
    const int D = m->c.d_model, qh = d.qh(), vh = pad8(d.vdim);
    const bool kv = L.own_kv();
    const HostTensor *q, *g, *k = nullptr, *v = nullptr, *o, *t;
    DEC_TRY(want_tensor(m, pre + "mix.q", d.H * d.dim, D, &q));
    DEC_TRY(want_tensor(m, pre + "mix.g", d.H, D, &g));
    DEC_TRY(want_tensor(m, pre + "mix.o", D, d.H * d.vdim, &o));
    if (kv) {
        DEC_TRY(want_tensor(m, pre + "mix.k", d.G * d.dim, D, &k));
        DEC_TRY(want_tensor(m, pre + "mix.v", d.G * d.vdim, D, &v));
    }
    {
        HostMatrix h(m->f32, d.wide_cols(kv), m->wp);
        put_heads(h, 0, *q, d.H, d.dim, qh);
        for (int i = 0; i < d.H; ++i) h.put_row(d.q_cols() + i, *g, i);
        if (kv) {
            put_heads(h, d.q_cols() + pad8(d.H), *k, d.G, d.dim, qh);
            put_heads(h, d.q_cols() + pad8(d.H) + d.G * qh, *v, d.G, d.vdim, vh);
        }
        DEC_TRY(upload_proj(m, h, &L.qd));
    }
    {
        HostMatrix h(m->f32, m->wp, d.out_cols());
        for (int j = 0; j < D; ++j) h.put_row(j, *o, j);
        DEC_TRY(upload_proj(m, h, &L.out));
    }
    DEC_TRY(want_tensor(m, pre + "mix.q.b", d.H * d.dim, 1, &t));
    DEC_TRY(upload_heads(m, *t, d.H, d.dim, qh, &L.aw.q_bias));
    DEC_TRY(want_tensor(m, pre + "mix.q.norm", d.dim, 1, &t));
    DEC_TRY(upload_vec(m, *t, qh, &L.aw.q_norm));
    DEC_TRY(want_tensor(m, pre + "mix.sink", d.H, 1, &t));
    DEC_TRY(upload_vec(m, *t, pad8(d.H), &L.aw.sink));
    if (kv) {
        DEC_TRY(want_tensor(m, pre + "mix.k.b", d.G * d.dim, 1, &t));
        DEC_TRY(upload_heads(m, *t, d.G, d.dim, qh, &L.aw.k_bias));
        DEC_TRY(want_tensor(m, pre + "mix.k.norm", d.dim, 1, &t));
        DEC_TRY(upload_vec(m, *t, qh, &L.aw.k_norm));
        DEC_TRY(want_tensor(m, pre + "mix.v.b", d.G * d.vdim, 1, &t));
        DEC_TRY(upload_heads(m, *t, d.G, d.vdim, vh, &L.aw.v_bias));
    }
    return JSM_OK;
}

static jsm_status build_recurrence(jsm_decoder* m, DecLayer& L, const std::string& pre) {
    const RecDims& d = L.rd;
    const int D = m->c.d_model, kp = d.kp(), vp = d.vp(), cc = d.conv_cols();
    const HostTensor *q, *k, *v, *z, *o, *t;
    DEC_TRY(want_tensor(m, pre + "mix.q", d.G * d.dk, D, &q));
    DEC_TRY(want_tensor(m, pre + "mix.k", d.G * d.dk, D, &k));
    DEC_TRY(want_tensor(m, pre + "mix.v", d.H * d.dv, D, &v));
    DEC_TRY(want_tensor(m, pre + "mix.g", d.H * d.dv, D, &z));
    DEC_TRY(want_tensor(m, pre + "mix.o", D, d.H * d.dv, &o));
    {
        HostMatrix h(m->f32, d.raw_cols(), m->wp);
        put_heads(h, 0, *q, d.G, d.dk, kp);
        put_heads(h, d.G * kp, *k, d.G, d.dk, kp);
        put_heads(h, 2 * d.G * kp, *v, d.H, d.dv, vp);
        put_heads(h, cc, *z, d.H, d.dv, vp);
        DEC_TRY(upload_proj(m, h, &L.in));
    }
    {
        HostMatrix h(m->f32, m->wp, d.out_cols());
        for (int r = 0; r < D; ++r)
            for (int i = 0; i < d.H; ++i)
                for (int j = 0; j < d.dv; ++j) h.set(r, i * vp + j, o->at((long long)r * d.H * d.dv + i * d.dv + j));
        DEC_TRY(upload_proj(m, h, &L.out));
    }
    {
        HostMatrix c(true, d.taps, cc);
        if (d.delta) {
            const std::pair<const char*, int> parts[3] = {{"mix.q.conv", d.G * d.dk}, {"mix.k.conv", d.G * d.dk}, {"mix.v.conv", d.H * d.dv}};
            for (int p = 0; p < 3; ++p) {
                DEC_TRY(want_tensor(m, pre + parts[p].first, parts[p].second, d.taps, &t));
                const int dim = p < 2 ? d.dk : d.dv, pitch = p < 2 ? kp : vp, at = p * d.G * kp;
                for (int j = 0; j < parts[p].second; ++j)
                    for (int n = 0; n < d.taps; ++n) c.set(n, at + j / dim * pitch + j % dim, t->at((long long)j * d.taps + n));
            }
        } else {
            for (int j = 0; j < cc; ++j) c.set(0, j, 1.0f);  // no convolution: its activation alone
        }
        void* p = nullptr;
        DEC_TRY(upload_plain(m, c, &p));
        L.rw.conv = static_cast<float*>(p);
    }
    if (!d.delta) {
        DEC_TRY(want_tensor(m, pre + "mix.norm", d.H * d.dv, 1, &t));
        DEC_TRY(upload_heads(m, *t, d.H, d.dv, vp, &L.rw.norm));
        DEC_TRY(want_tensor(m, pre + "mix.decay", d.H, 1, &t));
        HostTensor lg;
        lg.rows = d.H; lg.cols = 1;
        for (int i = 0; i < d.H; ++i) {
            const float g = t->at(i);
            if (!(g >= 0.0f && g <= 1.0f)) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder: '%smix.decay' holds %g", pre.c_str(), g);
            lg.v.push_back(g > 0.0f ? (float)log((double)g) : -1.0e30f);
        }
        DEC_TRY(upload_vec(m, *t, pad8(d.H), &L.rw.decay));
        return upload_vec(m, lg, pad8(d.H), &L.rw.log_decay);
    }
    DEC_TRY(want_tensor(m, pre + "mix.norm", d.dv, 1, &t));
    DEC_TRY(upload_vec(m, *t, vp, &L.rw.norm));
    DEC_TRY(want_tensor(m, pre + "mix.dt_bias", d.H, 1, &t));
    DEC_TRY(upload_vec(m, *t, pad8(d.H), &L.rw.dt_bias));
    DEC_TRY(want_tensor(m, pre + "mix.A_log", d.H, 1, &t));
    HostTensor A;
    A.rows = d.H; A.cols = 1;
    for (int i = 0; i < d.H; ++i) A.v.push_back((float)-exp((double)t->at(i)));
    DEC_TRY(upload_vec(m, A, pad8(d.H), &L.rw.A));
    const HostTensor *b, *a;
    DEC_TRY(want_tensor(m, pre + "mix.b", d.H, D, &b));
    DEC_TRY(want_tensor(m, pre + "mix.a", d.H, D, &a));
    HostMatrix h(m->f32, d.ba_cols(), m->wp);
    for (int i = 0; i < d.H; ++i) {
        h.put_row(i, *b, i);
        h.put_row(d.ba_cols() / 2 + i, *a, i);
    }
    DEC_TRY(upload_proj(m, h, &L.xp));
    if (!m->f32) DEC_TRY(upload_plain(m, h, &L.xp.rows));
    L.rw.ba = m->f32 ? (void*)L.xp.w32 : L.xp.rows;
    return JSM_OK;
}

static jsm_status build_mixer(jsm_decoder* m, DecLayer& L, const std::string& pre) {
    switch (L.c.mixer) {
        case JSM_MIXER_LATENT_ATTENTION: return build_latent(m, L, pre);
        case JSM_MIXER_SELECTIVE_SCAN: return build_scan(m, L, pre);
        case JSM_MIXER_ATTENTION: return build_attention(m, L, pre);
        default: return build_recurrence(m, L, pre);
    }
}

static jsm_status build_ff(jsm_decoder* m, DecLayer& L, const std::string& pre) {
    const int D = m->c.d_model, F = L.c.ff, fp = L.ffp();
    const HostTensor *g, *u, *w;
    DEC_TRY(want_tensor(m, pre + "mlp.gate", F, D, &g));
    DEC_TRY(want_tensor(m, pre + "mlp.up", F, D, &u));
    DEC_TRY(want_tensor(m, pre + "mlp.down", D, F, &w));
    if (m->f32) {
        HostMatrix hg(true, fp, m->wp), hu(true, fp, m->wp);
        for (int j = 0; j < F; ++j) { hg.put_row(j, *g, j); hu.put_row(j, *u, j); }
        DEC_TRY(upload_proj(m, hg, &L.gate));
        DEC_TRY(upload_proj(m, hu, &L.up));
    } else {
        HostMatrix h(false, 2 * fp, m->wp);
        for (int j = 0; j < F; ++j) { h.put_row(j, *g, j); h.put_row(fp + j, *u, j); }
        DEC_TRY(upload_proj(m, h, &L.gate, true));
    }
    HostMatrix h(m->f32, m->wp, fp);
    for (int j = 0; j < D; ++j) h.put_row(j, *w, j);
    return upload_proj(m, h, &L.down);
}

// Y = X . W^T; X act [T][x_stride], Y f32 (out_f32) or act [T][N]
static jsm_status linear(jsm_decoder* m, const Proj& p, const void* X, long long x_stride, void* Y, bool out_f32, int T, cudaStream_t st,
                         float glu_limit = 0.0f, int glu = LIN_CLAMPED_GLU) {
    if (m->f32) {
        jsm_mat A{const_cast<void*>(X), T, p.K, x_stride, 1, JSM_F32};
        jsm_mat B{p.w32, p.K, p.N, 1, p.K, JSM_F32};
        jsm_mat C{Y, T, p.N, p.N, 1, JSM_F32};
        return dot_f32_launch(A, B, C, st);
    }
    PackedArgs a;
    a.Wp = p.packed; a.bias = nullptr; a.R = nullptr; a.out_f32 = out_f32;
    a.epilogue = p.paired ? glu : LIN_NONE;
    a.glu_alpha = GLU_ALPHA; a.glu_limit = glu_limit;
    a.N = p.N; a.K = p.K; a.x_row_stride = x_stride;
    a.ws = m->ws; a.ws_floats = m->ws_floats; a.counters = m->counters; a.n_counters = m->n_counters;
    a.chained = true;  // the weights are constant while the model's stream runs
    if (p.rows && T > 64 && x_stride == p.K) {
        // the packed kernel streams the weights once per 256 tokens over all SMs, which suits wide and deep matrices; here one
        // launch tiles outputs x tokens, split along K while that leaves SMs idle
        const int tiles = ((p.N + 127) / 128) * ((T + 127) / 128);
        LinearArgs r;
        r.X = X; r.W = p.rows; r.bias = nullptr; r.epilogue = LIN_NONE; r.R = nullptr; r.Y = Y;
        r.out_mode = out_f32 ? 1 : 0;
        r.T = T; r.N = p.N; r.K = p.K; r.impl = 2;
        r.splits = std::max(1, std::min(sm_count() / tiles, p.K / 512));
        r.ws = r.splits > 1 ? m->ws : nullptr;
        r.counters = m->counters;
        r.chained = true;
        return linear_bf16_launch(r, st);
    }
    for (int t0 = 0; t0 < T; t0 += 256) {
        a.T = std::min(256, T - t0);
        a.X = static_cast<const __nv_bfloat16*>(X) + (long long)t0 * x_stride;
        a.Y = out_f32 ? static_cast<void*>(static_cast<float*>(Y) + (long long)t0 * p.N)
                      : static_cast<void*>(static_cast<__nv_bfloat16*>(Y) + (long long)t0 * p.N);
        DEC_TRY(linear_packed_launch(a, st));
    }
    return JSM_OK;
}

// ---- one pass -----------------------------------------------------------------------------------------------------
struct TileList { size_t seg_off, r0_off; int n, tokens; };
struct Pass {
    StepTokens tk;
    int n_flash = 0;           // the last n_flash segments are long
    std::vector<PassSeg> segs; // short segments first
    std::vector<int> starts;   // first token of each segment within the pass
    const int32_t* want = nullptr;
    int n_want = 0;
    bool decode = false;       // one token per segment
    std::map<std::pair<int, int>, TileList> tiles_short, tiles_all;  // per (rows per token, rows per tile)
    RecChunks chunks;          // of the passes that are no decode steps
    int32_t* meta = nullptr;
};

static jsm_status latent_mixer(jsm_decoder* m, DecLayer& L, const Pass& P, cudaStream_t st) {
    const LatentDims& d = L.ld;
    const int T = P.tk.T;
    const void* xin = m->f32 ? m->x : m->xa;
    DEC_TRY(linear(m, L.qd, xin, m->wp, m->wide, true, T, st));
    const bool flash = L.expand.packed != nullptr && P.n_flash > 0;
    const TileList& tl = (flash ? P.tiles_short : P.tiles_all).at(L.tiling(P.decode));
    DEC_TRY(latent_prep_launch(m->f32, m->wide, d, L.lw, m->c.norm_eps, L.cache, P.tk, m->q, tl.n > 0 ? m->q_lat : nullptr, st));
    if (tl.n > 0) {
        LatentTiles t;
        t.tile_seg = P.meta + tl.seg_off; t.tile_r0 = P.meta + tl.r0_off; t.n_tiles = tl.n; t.t_first = 0; t.t_count = tl.tokens;
        t.max_keys = std::min(d.window, m->c.max_context);
        LatentScratch sc{m->q_lat, m->o_lat, m->part, m->part_floats};
        DEC_TRY(latent_attn_launch(m->f32, d, L.lw, L.cache, P.tk, t, m->q, sc, m->att, st));
    }
    if (flash) {
        for (size_t i = P.segs.size() - P.n_flash; i < P.segs.size(); ++i) {
            const PassSeg& s = P.segs[i];
            const int k0 = std::max(0, s.pos0 - d.window + 1), n = s.pos0 + s.len - k0;
            DEC_TRY(latent_gather_launch(d, L.cache, s.row, k0, n, m->gathered, st));
            DEC_TRY(linear(m, L.expand, m->gathered, d.cr(), m->expanded, false, n, st));
            const __nv_bfloat16* k = static_cast<const __nv_bfloat16*>(m->expanded);
            DEC_TRY(latent_flash_launch(d, static_cast<const __nv_bfloat16*>(m->q) + (long long)P.starts[i] * d.q_cols(), k, k + d.H * d.dkp(),
                                        L.expand.N, static_cast<__nv_bfloat16*>(m->att) + (long long)P.starts[i] * d.out_cols(), s.len, n, st));
        }
    }
    return linear(m, L.out, m->att, d.out_cols(), m->y, true, T, st);
}

static jsm_status scan_mixer(jsm_decoder* m, DecLayer& L, const Pass& P, cudaStream_t st) {
    const ScanDims& d = L.sd;
    const int T = P.tk.T;
    const void* xin = m->f32 ? m->x : m->xa;
    DEC_TRY(linear(m, L.in, xin, m->wp, m->xz, false, T, st));
    DEC_TRY(scan_conv_launch(m->f32, d, L.sw, L.state, P.tk, m->xz, m->xc, P.decode, st));
    DEC_TRY(linear(m, L.xp, m->xc, d.ip(), m->proj, true, T, st));
    if (P.decode) {
        DEC_TRY(scan_step_launch(m->f32, d, L.sw, L.state, P.tk, m->xz, m->xc, m->proj, m->scan_y, st));
    } else {
        if (m->f32) {
            DEC_TRY(linear(m, L.dt, m->proj, d.proj_cols(), m->dt_raw, true, T, st));
        } else {
            DEC_TRY(scan_dt_operand_launch(d, m->proj, m->dt_op, T, st));
            DEC_TRY(linear(m, L.dt, m->dt_op, d.rp(), m->dt_raw, true, T, st));
        }
        DEC_TRY(scan_launch(m->f32, d, L.sw, L.state, P.tk, m->xz, m->xc, m->proj, m->dt_raw, m->scan_y, st));
    }
    return linear(m, L.out, m->scan_y, d.ip(), m->y, true, T, st);
}

static jsm_status attention_mixer(jsm_decoder* m, DecLayer& L, const Pass& P, cudaStream_t st) {
    const AttnDims& d = L.ad;
    const int T = P.tk.T;
    DEC_TRY(linear(m, L.qd, m->f32 ? m->x : m->xa, m->wp, m->wide, true, T, st));
    DEC_TRY(attn_prep_launch(m->f32, m->wide, d, L.aw, m->c.norm_eps, L.ac, L.own_kv(), P.tk, m->q, m->head_gate, st));
    const bool flash = !m->f32 && P.n_flash > 0 && attn_flash_usable(d);
    const std::pair<int, int> shape = L.tiling(P.decode);
    const TileList& tl = (flash ? P.tiles_short : P.tiles_all).at(shape);
    if (tl.n > 0) {
        const AttnTiles t{P.meta + tl.seg_off, P.meta + tl.r0_off, tl.n, shape.second, 0, tl.tokens, d.mask.reach(m->c.max_context)};
        DEC_TRY(attn_paged_launch(m->f32, d, L.aw, L.ac, P.tk, t, m->q, m->head_gate, AttnScratch{m->part, m->part_floats, m->attn_ctrs, attn_counters()},
                                  m->att, st));
    }
    if (flash)
        for (size_t i = P.segs.size() - P.n_flash; i < P.segs.size(); ++i) {
            const PassSeg& s = P.segs[i];
            DEC_TRY(attn_flash_launch(d, L.aw, L.ac, s.row, s.pos0, s.len, static_cast<const __nv_bfloat16*>(m->q) + (long long)P.starts[i] * d.q_cols(),
                                      m->head_gate + (long long)P.starts[i] * d.H, static_cast<__nv_bfloat16*>(m->att) + (long long)P.starts[i] * d.out_cols(),
                                      st));
        }
    return linear(m, L.out, m->att, d.out_cols(), m->y, true, T, st);
}

static jsm_status recurrence_mixer(jsm_decoder* m, DecLayer& L, const Pass& P, cudaStream_t st) {
    const RecDims& d = L.rd;
    const int T = P.tk.T;
    const void* xin = m->f32 ? m->x : m->xa;
    DEC_TRY(linear(m, L.in, xin, m->wp, m->xz, false, T, st));
    DEC_TRY(short_conv_launch(m->f32, m->xz, d.raw_cols(), d.conv_cols(), d.taps, L.rw.conv, nullptr, L.rs.conv, P.tk, m->xc, P.decode, st));
    if (P.decode) {
        DEC_TRY(rec_step_launch(m->f32, d, L.rw, L.rs, m->c.norm_eps, P.tk, m->xz, m->xc, xin, m->wp, m->scan_y, st));
    } else {
        if (d.delta) DEC_TRY(linear(m, L.xp, xin, m->wp, m->proj, true, T, st));
        DEC_TRY(rec_scan_launch(m->f32, d, L.rw, L.rs, m->c.norm_eps, P.tk, P.chunks, m->xz, m->xc, m->proj, m->scan_y, st));
        DEC_TRY(short_conv_carry_launch(m->f32, m->xz, d.raw_cols(), d.conv_cols(), d.taps, L.rs.conv, P.tk, st));
    }
    return linear(m, L.out, m->scan_y, d.out_cols(), m->y, true, T, st);
}

static jsm_status run_mixer(jsm_decoder* m, DecLayer& L, const Pass& P, cudaStream_t st) {
    switch (L.c.mixer) {
        case JSM_MIXER_LATENT_ATTENTION: return latent_mixer(m, L, P, st);
        case JSM_MIXER_SELECTIVE_SCAN: return scan_mixer(m, L, P, st);
        case JSM_MIXER_ATTENTION: return attention_mixer(m, L, P, st);
        default: return recurrence_mixer(m, L, P, st);
    }
}

// a sublayer's output y joins the residual stream
static jsm_status join_residual(jsm_decoder* m, const float* gain, int T, cudaStream_t st) {
    const jsm_decoder_config& c = m->c;
    return c.norm_place == JSM_NORM_SUM ? sum_norm_launch(m->y, m->x, gain, c.norm_eps, c.residual_scale, m->xa, T, c.d_model, m->wp, st)
                                        : post_norm_add_launch(m->y, m->x, gain, c.norm_eps, m->xa, T, c.d_model, m->wp, st);
}

static jsm_status run_layers(jsm_decoder* m, const Pass& P, cudaStream_t st) {
    const int T = P.tk.T, D = m->c.d_model, wp = m->wp;
    DEC_TRY(embed_residual_launch(m->f32, m->embed, P.tk.ids, m->c.embed_scale, m->x, m->xa, T, wp, st));
    for (size_t l = 0; l < m->layers.size(); ++l) {
        DecLayer& L = m->layers[l];
        DEC_TRY(run_mixer(m, L, P, st));
        DEC_TRY(join_residual(m, L.norm1, T, st));
        if (L.c.ff > 0) {
            const void* xin = m->f32 ? m->x : m->xa;
            if (m->f32) {
                float* up = m->gate32 + (size_t)m->c.max_step_tokens * L.ffp();
                DEC_TRY(linear(m, L.gate, xin, wp, m->gate32, true, T, st));
                DEC_TRY(linear(m, L.up, xin, wp, up, true, T, st));
                if (L.c.ff_kind == JSM_FF_GELU_GLU) DEC_TRY(gelu_glu_f32_launch(m->gate32, up, static_cast<float*>(m->act), (long long)T * L.ffp(), st));
                else DEC_TRY(clamped_glu_f32_launch(m->gate32, up, static_cast<float*>(m->act), GLU_ALPHA, L.c.ff_limit, (long long)T * L.ffp(), st));
            } else {
                DEC_TRY(linear(m, L.gate, xin, wp, m->act, false, T, st, L.c.ff_limit, L.c.ff_kind == JSM_FF_GELU_GLU ? LIN_GELU_GLU : LIN_CLAMPED_GLU));
            }
            DEC_TRY(linear(m, L.down, m->act, L.ffp(), m->y, true, T, st));
            DEC_TRY(join_residual(m, L.norm2, T, st));
        }
        if (m->tap)
            JSM_CUDA_CHECK(cudaMemcpy2DAsync(m->tap + l * (size_t)T * D, sizeof(float) * D, m->x, sizeof(float) * wp, sizeof(float) * D, T,
                                             cudaMemcpyDeviceToDevice, st));
    }
    return JSM_OK;
}

// logits and arg-max of wanted rows [w0, w0 + n) of the pass into the logits buffer
static jsm_status run_head(jsm_decoder* m, const Pass& P, int w0, int n, cudaStream_t st) {
    DEC_TRY(final_norm_launch(m->f32, m->x, P.want + w0, m->final_norm, m->c.norm_eps, m->head_in, n, m->c.d_model, m->wp, st));
    DEC_TRY(linear(m, m->head, m->head_in, m->wp, m->logits, true, n, st));
    return logits_finish_launch(m->logits, m->vp, m->c.vocab, m->c.logit_softcap, n, m->keys, m->key_ctrs, m->next_dev, st);
}

// first position that a token at `pos` or later can see in any layer
static int first_needed(const jsm_decoder* m, int pos) {
    int first = pos;
    for (const DecLayer& L : m->layers)
        if (L.is_attention()) first = std::min(first, L.key_mask().first(pos));
    return first;
}

// Runs the tokens of `segs`; want_tok / want_out: wanted places as (flat token, output row) pairs.
static jsm_status run_pass(jsm_decoder* m, std::vector<PassSeg> segs, const int32_t* h_ids, const std::vector<std::pair<int, int>>& want,
                           int32_t* h_next, float* h_logits, cudaStream_t st) {
    Pass P;
    std::stable_sort(segs.begin(), segs.end(), [](const PassSeg& a, const PassSeg& b) { return (a.len >= FLASH_MIN_TOKENS) < (b.len >= FLASH_MIN_TOKENS); });
    P.segs = segs;
    const int E = (int)segs.size();
    int T = 0, max_len = 0, tok_short = 0;
    for (const PassSeg& s : segs) {
        P.starts.push_back(T);
        T += s.len;
        max_len = std::max(max_len, s.len);
        if (s.len >= FLASH_MIN_TOKENS) ++P.n_flash;
        else tok_short = T;
        if (m->has_attention) DEC_TRY(m->rows.provision(s.row, s.pos0 + s.len, st));
    }
    P.decode = max_len == 1;
    P.n_want = (int)want.size();
    // metadata: one pinned buffer, one copy
    std::vector<int32_t> M;
    auto push = [&](int32_t v) { M.push_back(v); };
    for (const PassSeg& s : segs)
        for (int j = 0; j < s.len; ++j) push(h_ids[s.tok0 + j]);
    for (const PassSeg& s : segs)
        for (int j = 0; j < s.len; ++j) push(s.row);
    for (const PassSeg& s : segs)
        for (int j = 0; j < s.len; ++j) push(s.pos0 + j);
    const size_t seg_off = M.size();
    for (int i = 0; i < E; ++i) push(P.starts[i]);
    for (const PassSeg& s : segs) push(s.len);
    for (const PassSeg& s : segs) push(s.pos0);
    for (const PassSeg& s : segs) push(s.row);
    for (const PassSeg& s : segs) push(m->slot_of_row[s.row]);
    const size_t want_off = M.size();
    for (const auto& w : want) {
        for (int i = 0; i < E; ++i)
            if (w.first >= segs[i].tok0 && w.first < segs[i].tok0 + segs[i].len) push(P.starts[i] + (w.first - segs[i].tok0));
    }
    for (const DecLayer& L : m->layers) {
        if (!L.is_attention() || P.tiles_all.count(L.tiling(P.decode))) continue;
        const auto [H, rows] = L.tiling(P.decode);
        std::vector<int32_t> sg, r0;
        int n_short = 0;
        for (int i = 0; i < E; ++i) {
            for (long long r = 0; r < (long long)segs[i].len * H; r += rows) { sg.push_back(i); r0.push_back((int32_t)r); }
            if (i + 1 == E - P.n_flash) n_short = (int)sg.size();
        }
        const size_t so = M.size();
        M.insert(M.end(), sg.begin(), sg.end());
        const size_t ro = M.size();
        M.insert(M.end(), r0.begin(), r0.end());
        P.tiles_all[{H, rows}] = TileList{so, ro, (int)sg.size(), T};
        P.tiles_short[{H, rows}] = TileList{so, ro, n_short, tok_short};
    }
    const size_t chunk_off = M.size();
    if (m->chunk_bytes > 0 && !P.decode) {
        std::vector<int32_t> seg, t0, first;
        for (int i = 0; i < E; ++i) {
            first.push_back((int32_t)seg.size());
            for (int t = 0; t < segs[i].len; t += REC_CHUNK) { seg.push_back(i); t0.push_back(t); }
        }
        P.chunks.n_chunks = (int)seg.size();
        for (const auto* v : {&seg, &t0, &first}) M.insert(M.end(), v->begin(), v->end());
    }
    if (M.size() > m->meta_cap) JSM_FAIL(JSM_SHAPE, "jsm_decoder: step metadata of %zu words (room for %zu)", M.size(), m->meta_cap);
    memcpy(m->h_meta, M.data(), M.size() * sizeof(int32_t));
    JSM_CUDA_CHECK(cudaMemcpyAsync(m->meta, m->h_meta, M.size() * sizeof(int32_t), cudaMemcpyHostToDevice, st));
    P.meta = m->meta;
    P.tk.T = T; P.tk.n_segs = E; P.tk.max_len = max_len;
    P.tk.ids = m->meta; P.tk.tok_row = m->meta + T; P.tk.tok_pos = m->meta + 2 * T;
    P.tk.seg_start = m->meta + seg_off; P.tk.seg_len = P.tk.seg_start + E; P.tk.seg_pos0 = P.tk.seg_len + E;
    P.tk.seg_row = P.tk.seg_pos0 + E; P.tk.seg_slot = P.tk.seg_row + E;
    P.want = m->meta + want_off;
    P.chunks.chunk_seg = m->meta + chunk_off; P.chunks.chunk_t0 = P.chunks.chunk_seg + P.chunks.n_chunks;
    P.chunks.seg_chunk0 = P.chunks.chunk_t0 + P.chunks.n_chunks;
    P.chunks.ws = m->chunk_ws;

    const int n_head = std::min(P.n_want, m->cap_rows);
    const bool graph = P.decode && !m->tap && (P.n_want == 0 || (P.n_want == E && E <= m->cap_rows));
    if (graph) {
        const int key = 2 * E + (P.n_want ? 1 : 0);
        auto it = m->graphs.find(key);
        if (it == m->graphs.end()) {
            cudaGraph_t g = nullptr;
            JSM_CUDA_CHECK(cudaStreamBeginCapture(st, cudaStreamCaptureModeRelaxed));
            jsm_status s = run_layers(m, P, st);
            if (s == JSM_OK && P.n_want) s = run_head(m, P, 0, n_head, st);
            cudaError_t e = cudaStreamEndCapture(st, &g);
            if (s != JSM_OK) { if (g) cudaGraphDestroy(g); return s; }
            if (e != cudaSuccess) { cudaGetLastError(); JSM_FAIL(JSM_CUDA, "jsm_decoder: stream capture failed: %s", cudaGetErrorString(e)); }
            cudaGraphExec_t exec = nullptr;
            e = cudaGraphInstantiate(&exec, g, 0);
            cudaGraphDestroy(g);
            if (e != cudaSuccess) { cudaGetLastError(); JSM_FAIL(JSM_CUDA, "jsm_decoder: graph instantiation failed: %s", cudaGetErrorString(e)); }
            it = m->graphs.emplace(key, exec).first;
        }
        JSM_CUDA_CHECK(cudaGraphLaunch(it->second, st));
    } else {
        DEC_TRY(run_layers(m, P, st));
    }
    for (int w0 = 0; w0 < P.n_want; w0 += n_head) {
        const int n = std::min(n_head, P.n_want - w0);
        if (!graph) DEC_TRY(run_head(m, P, w0, n, st));
        for (int i = 0; i < n;) {  // runs of consecutive output rows
            int j = i + 1;
            while (j < n && want[w0 + j].second == want[w0 + j - 1].second + 1) ++j;
            const int out = want[w0 + i].second;
            if (h_next) JSM_CUDA_CHECK(cudaMemcpyAsync(h_next + out, m->next_dev + i, sizeof(int32_t) * (j - i), cudaMemcpyDeviceToHost, st));
            if (h_logits)
                JSM_CUDA_CHECK(cudaMemcpy2DAsync(h_logits + (size_t)out * m->c.vocab, sizeof(float) * m->c.vocab, m->logits + (size_t)i * m->vp,
                                                 sizeof(float) * m->vp, sizeof(float) * m->c.vocab, j - i, cudaMemcpyDeviceToHost, st));
            i = j;
        }
    }
    DEC_TRY(tc_check_error(st, "jsm_decoder_step"));  // synchronises: the metadata buffer is free, the outputs are valid
    JSM_CUDA_CHECK(cudaStreamSynchronize(st));
    for (const PassSeg& s : segs) {
        m->rows.h_ctx[s.row] = s.pos0 + s.len;
        if (m->has_attention) m->rows.release_before(s.row, first_needed(m, s.pos0 + s.len));
    }
    return JSM_OK;
}

}  // namespace jsm

using namespace jsm;

extern "C" {

jsm_status jsm_decoder_create(const jsm_decoder_config* cfg, const jsm_layer_config* layers, jsm_decoder** out) {
    if (!cfg || !layers || !out) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: null argument");
    *out = nullptr;
    const jsm_decoder_config& c = *cfg;
    if (c.n_layers <= 0 || c.d_model <= 0 || c.vocab <= 0 || c.max_batch <= 0 || c.max_context <= 0 || c.max_step_tokens <= 0 || c.n_pages < 0)
        JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: non-positive dimension");
    if (c.dtype != JSM_F32 && c.dtype != JSM_BF16) JSM_FAIL(JSM_UNSUPPORTED, "jsm_decoder_create: dtype %d", c.dtype);
    if (c.max_step_tokens < c.max_batch) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: %d tokens per step for %d rows", c.max_step_tokens, c.max_batch);
    for (int l = 0; l < c.n_layers; ++l) {
        const jsm_layer_config& k = layers[l];
        if (k.weights_of >= c.n_layers || (k.weights_of >= 0 && (k.weights_of == l || layers[k.weights_of].weights_of >= 0 || layers[k.weights_of].mixer != k.mixer)))
            JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: layer %d takes the weights of layer %d", l, k.weights_of);
        if (k.mixer == JSM_MIXER_LATENT_ATTENTION) {
            if (k.heads <= 0 || k.dim <= 0 || k.rot_dim < 0 || k.rot_dim % 2 || k.vdim <= 0 || k.kv_rank <= 0 || k.window <= 0 || !(k.rope_base > 0.0))
                JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: sizes of the latent attention of layer %d", l);
        } else if (k.mixer == JSM_MIXER_SELECTIVE_SCAN) {
            if (k.inner <= 0 || k.state <= 0 || k.dt_rank <= 0 || k.taps <= 0) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: sizes of the scan of layer %d", l);
            if (k.state > 128) JSM_FAIL(JSM_UNSUPPORTED, "jsm_decoder_create: %d states per channel in layer %d (at most 128)", k.state, l);
        } else if (k.mixer == JSM_MIXER_ATTENTION) {
            if (k.heads <= 0 || k.kv_heads <= 0 || k.heads % k.kv_heads || k.dim <= 0 || k.vdim <= 0 || k.rot_dim < 0 || k.rot_dim % 2 || k.rot_dim > k.dim ||
                (k.rot_dim > 0 && !(k.rope_base > 0.0)) || k.mask < JSM_MASK_FULL || k.mask > JSM_MASK_CHUNK || (k.mask != JSM_MASK_FULL && k.window <= 0))
                JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: sizes of the attention of layer %d", l);
            if (k.kv_from >= 0) {
                const jsm_layer_config& s = layers[std::min(k.kv_from, l)];
                if (k.kv_from >= l || s.mixer != JSM_MIXER_ATTENTION || s.kv_from >= 0 || s.heads != k.heads || s.kv_heads != k.kv_heads || s.dim != k.dim || s.vdim != k.vdim)
                    JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: layer %d takes the keys and values of layer %d", l, k.kv_from);
            }
        } else if (k.mixer == JSM_MIXER_LINEAR_ATTENTION || k.mixer == JSM_MIXER_DELTA) {
            const bool delta = k.mixer == JSM_MIXER_DELTA;
            if (k.heads <= 0 || k.dim <= 0 || k.vdim <= 0 || (delta && (k.kv_heads <= 0 || k.heads % k.kv_heads || k.taps <= 0)))
                JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: sizes of the recurrence of layer %d", l);
            if (!rec_usable(RecDims{k.heads, k.heads, k.dim, k.vdim, 1, delta}))
                JSM_FAIL(JSM_UNSUPPORTED, "jsm_decoder_create: recurrence of layer %d with heads of %d / %d components", l, k.dim, k.vdim);
        } else {
            JSM_FAIL(JSM_UNSUPPORTED, "jsm_decoder_create: mixer %d of layer %d", k.mixer, l);
        }
        if (k.ff < 0 || k.ff_kind < JSM_FF_CLAMPED_GLU || k.ff_kind > JSM_FF_GELU_GLU) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_create: feed-forward of layer %d", l);
    }
    if (c.norm_place != JSM_NORM_OUTPUT && c.norm_place != JSM_NORM_SUM) JSM_FAIL(JSM_UNSUPPORTED, "jsm_decoder_create: norm place %d", c.norm_place);
    int ndev = 0;
    DEC_TRY(jsm_device_count(&ndev));
    if (ndev == 0) JSM_FAIL(JSM_CUDA, "jsm_decoder_create: no CUDA device");
    jsm_decoder* m = new jsm_decoder();
    m->c = c;
    if (m->c.embed_scale == 0.0f) m->c.embed_scale = 1.0f;
    m->f32 = c.dtype == JSM_F32;
    m->wp = pad8(c.d_model);
    m->vp = pad8(c.vocab);
    m->layers.resize(c.n_layers);
    for (int l = 0; l < c.n_layers; ++l) {
        DecLayer& L = m->layers[l];
        L.c = layers[l];
        if (L.c.mixer == JSM_MIXER_LATENT_ATTENTION) {
            L.ld = LatentDims{L.c.heads, L.c.dim, L.c.rot_dim, L.c.vdim, L.c.kv_rank, L.c.window, (float)L.c.scale};
        } else if (L.c.mixer == JSM_MIXER_ATTENTION) {
            L.ad = AttnDims{L.c.heads, L.c.kv_heads, L.c.dim, L.c.vdim, L.c.rot_dim, KeyMask{L.c.mask, L.c.window}, (float)L.c.scale, 1};
        } else if (L.is_recurrence()) {
            const bool delta = L.c.mixer == JSM_MIXER_DELTA;
            L.rd = RecDims{L.c.heads, delta ? L.c.kv_heads : L.c.heads, L.c.dim, L.c.vdim, delta ? L.c.taps : 1, delta};
        } else {
            L.sd = ScanDims{L.c.inner, L.c.state, L.c.dt_rank, L.c.taps};
        }
    }
    for (const DecLayer& L : m->layers) m->has_attention |= L.is_attention();
    if (cudaStreamCreateWithFlags(&m->own_stream, cudaStreamNonBlocking) != cudaSuccess) {
        cudaGetLastError();
        delete m;
        JSM_FAIL(JSM_CUDA, "jsm_decoder_create: no stream");
    }
    *out = m;
    return JSM_OK;
}

jsm_status jsm_decoder_destroy(jsm_decoder* m) {
    if (!m) return JSM_OK;
    cudaDeviceSynchronize();
    for (auto& g : m->graphs) cudaGraphExecDestroy(g.second);
    for (void* p : m->allocs) cudaFree(p);
    if (m->h_meta) cudaFreeHost(m->h_meta);
    if (m->own_stream) cudaStreamDestroy(m->own_stream);
    delete m;
    return JSM_OK;
}

jsm_status jsm_decoder_set_weight(jsm_decoder* m, const char* name, const void* h_src, int dtype, int rows, int cols) {
    if (!m || !name || !h_src) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_set_weight: null argument");
    if (m->ready) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_set_weight: the model is already finalized");
    if (rows <= 0 || cols <= 0 || (dtype != JSM_F32 && dtype != JSM_BF16)) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_set_weight: '%s' [%d, %d], dtype %d", name, rows, cols, dtype);
    HostTensor& t = m->tensors[name];
    t = HostTensor();
    t.rows = rows; t.cols = cols;
    const size_t n = (size_t)rows * cols;
    if (dtype == JSM_F32) t.v.assign(static_cast<const float*>(h_src), static_cast<const float*>(h_src) + n);
    else t.b.assign(static_cast<const uint16_t*>(h_src), static_cast<const uint16_t*>(h_src) + n);
    return JSM_OK;
}

jsm_status jsm_decoder_finalize(jsm_decoder* m) {
    if (!m) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_finalize: null model");
    if (m->ready) return JSM_OK;
    const jsm_decoder_config& c = m->c;
    const int wp = m->wp;
    const size_t es = m->f32 ? 4 : 2;  // bytes per activation
    const HostTensor *emb, *fn;
    DEC_TRY(want_tensor(m, "embed", c.vocab, c.d_model, &emb));
    DEC_TRY(want_tensor(m, "final.norm", c.d_model, 1, &fn));
    {
        HostMatrix h(m->f32, m->vp, wp);
        for (int r = 0; r < c.vocab; ++r) h.put_row(r, *emb, r);
        DEC_TRY(upload_proj(m, h, &m->head));
        if (m->f32) m->embed = m->head.w32;
        else DEC_TRY(upload_plain(m, h, &m->embed));
    }
    DEC_TRY(upload_vec(m, *fn, wp, &m->final_norm));
    for (size_t l = 0; l < m->layers.size(); ++l) {
        DecLayer& L = m->layers[l];
        if (L.c.weights_of >= 0) continue;
        const std::string pre = "l" + std::to_string(l) + ".";
        const HostTensor* t;
        DEC_TRY(want_tensor(m, pre + "norm1", c.d_model, 1, &t));
        DEC_TRY(upload_vec(m, *t, wp, &L.norm1));
        DEC_TRY(build_mixer(m, L, pre));
        if (L.c.ff > 0) {
            DEC_TRY(want_tensor(m, pre + "norm2", c.d_model, 1, &t));
            DEC_TRY(upload_vec(m, *t, wp, &L.norm2));
            DEC_TRY(build_ff(m, L, pre));
        }
    }
    for (DecLayer& L : m->layers) {
        if (L.c.weights_of < 0) continue;
        const DecLayer& S = m->layers[L.c.weights_of];
        if ((L.c.ff > 0) != (S.c.ff > 0) || L.c.ff != S.c.ff) JSM_FAIL(JSM_SHAPE, "jsm_decoder_finalize: layers that share weights differ in their feed-forward");
        if (memcmp(&L.ld, &S.ld, offsetof(LatentDims, window)) != 0 || memcmp(&L.sd, &S.sd, sizeof(ScanDims)) != 0 ||
            memcmp(&L.ad, &S.ad, offsetof(AttnDims, mask)) != 0 || memcmp(&L.rd, &S.rd, offsetof(RecDims, delta)) != 0 || L.own_kv() != S.own_kv())
            JSM_FAIL(JSM_SHAPE, "jsm_decoder_finalize: layers that share weights differ in their sizes");
        L.norm1 = S.norm1; L.norm2 = S.norm2;
        L.qd = S.qd; L.expand = S.expand; L.in = S.in; L.xp = S.xp; L.dt = S.dt; L.out = S.out;
        L.gate = S.gate; L.up = S.up; L.down = S.down; L.lw = S.lw; L.sw = S.sw; L.aw = S.aw; L.rw = S.rw;
    }
    m->tensors.clear();
    // cache pages, states
    const int per_row = (c.max_context + JSM_PAGE_SIZE - 1) / JSM_PAGE_SIZE;
    const int n_pages = c.n_pages > 0 ? c.n_pages : c.max_batch * per_row;
    int32_t* bt = nullptr;
    DEC_TRY(dalloc(m, &bt, sizeof(int32_t) * (size_t)c.max_batch * per_row));
    m->rows.init(c.max_batch, n_pages, per_row, c.max_context, bt);
    m->slot_of_row.assign(c.max_batch, 0);
    for (int i = c.max_batch - 1; i >= 0; --i) m->free_slots.push_back(i);
    std::map<std::vector<double>, float2*> ropes;
    size_t wide = 0, q = 0, qlat = 0, olat = 0, att = 0, xz = 0, xc = 0, sy = 0, dtr = 0, proj = 0, rp = 0, ff = 0, part = 0, gat = 0, exp_cols = 0, gates = 0;
    auto rope_table = [&](const jsm_layer_config& k, const float2** out) -> jsm_status {
        *out = nullptr;
        if (k.rot_dim == 0) return JSM_OK;
        float2*& table = ropes[{(double)k.rot_dim, k.rope_base, k.rope_factor, k.rope_original, k.rope_fast, k.rope_slow}];
        if (!table) {
            DEC_TRY(dalloc(m, &table, sizeof(float2) * (size_t)c.max_context * (k.rot_dim / 2)));
            DEC_TRY(jsm_rope_scaled_table(reinterpret_cast<float*>(table), k.rot_dim, k.rope_base, k.rope_factor, k.rope_original, k.rope_fast, k.rope_slow,
                                          c.max_context));
        }
        *out = table;
        return JSM_OK;
    };
    for (DecLayer& L : m->layers) {
        if (L.c.mixer == JSM_MIXER_LATENT_ATTENTION) {
            const LatentDims& d = L.ld;
            DEC_TRY(dalloc(m, &L.cache.pool, (size_t)n_pages * JSM_PAGE_SIZE * d.cr() * es));
            L.cache.block_table = bt;
            L.cache.max_pages = per_row;
            DEC_TRY(rope_table(L.c, &L.cache.rope));
            wide = std::max(wide, (size_t)d.q_cols() + d.down_cols());
            q = std::max(q, (size_t)d.q_cols());
            qlat = std::max(qlat, (size_t)d.H * d.cr());
            olat = std::max(olat, (size_t)d.H * pad8(d.rank));
            att = std::max(att, (size_t)d.out_cols());
            part = std::max(part, latent_part_floats(d));
            if (L.expand.packed) {
                const int n = std::min(c.max_context, std::min(c.max_step_tokens, c.max_context) + d.window - 1);
                m->kv_rows = std::max(m->kv_rows, n);
                gat = std::max(gat, (size_t)d.cr());
                exp_cols = std::max(exp_cols, (size_t)L.expand.N);
            }
        } else if (L.c.mixer == JSM_MIXER_ATTENTION) {
            const AttnDims& d = L.ad;
            if (L.own_kv()) DEC_TRY(dalloc(m, &L.ac.pool, (size_t)n_pages * d.page_elems() * es));
            else L.ac.pool = m->layers[L.c.kv_from].ac.pool;
            L.ac.block_table = bt;
            L.ac.max_pages = per_row;
            DEC_TRY(rope_table(L.c, &L.ac.rope));
            wide = std::max(wide, (size_t)d.wide_cols(L.own_kv()));
            q = std::max(q, (size_t)d.q_cols());
            att = std::max(att, (size_t)d.out_cols());
            gates = std::max(gates, (size_t)d.H);
            if (attn_mma_usable(d)) part = std::max(part, attn_part_floats(d));
        } else if (L.is_recurrence()) {
            const RecDims& d = L.rd;
            DEC_TRY(dalloc(m, &L.rs.S, sizeof(float) * (size_t)c.max_batch * d.H * d.kp() * d.vp()));
            DEC_TRY(dalloc(m, &L.rs.conv, es * (size_t)c.max_batch * (d.taps - 1) * d.conv_cols()));
            xz = std::max(xz, (size_t)d.raw_cols());
            xc = std::max(xc, (size_t)d.conv_cols());
            sy = std::max(sy, (size_t)d.out_cols());
            proj = std::max(proj, (size_t)d.ba_cols());
            if (!m->f32 && rec_chunk_usable(d)) m->chunk_bytes = std::max(m->chunk_bytes, rec_chunk_bytes(d));
        } else {
            const ScanDims& d = L.sd;
            DEC_TRY(dalloc(m, &L.state.S, sizeof(float) * (size_t)c.max_batch * d.ip() * d.np()));
            DEC_TRY(dalloc(m, &L.state.conv, es * (size_t)c.max_batch * (d.taps - 1) * d.ip()));
            xz = std::max(xz, (size_t)2 * d.ip());
            xc = std::max(xc, (size_t)d.ip());
            sy = std::max(sy, (size_t)d.ip());
            dtr = std::max(dtr, (size_t)d.ip());
            proj = std::max(proj, (size_t)d.proj_cols());
            rp = std::max(rp, (size_t)d.rp());
        }
        ff = std::max(ff, (size_t)L.ffp());
    }
    const size_t T = c.max_step_tokens;
    m->cap_rows = std::max(c.max_batch, std::min(c.max_step_tokens, 256));
    DEC_TRY(dalloc(m, &m->x, 4 * T * wp));
    DEC_TRY(dalloc(m, &m->y, 4 * T * wp));
    if (!m->f32) DEC_TRY(dalloc(m, &m->xa, 2 * T * wp));
    DEC_TRY(dalloc(m, &m->wide, 4 * T * wide));
    DEC_TRY(dalloc(m, &m->q, es * T * q));
    DEC_TRY(dalloc(m, &m->q_lat, es * T * qlat));
    DEC_TRY(dalloc(m, &m->o_lat, es * T * olat));
    DEC_TRY(dalloc(m, &m->att, es * T * att));
    DEC_TRY(dalloc(m, &m->xz, es * T * xz));
    DEC_TRY(dalloc(m, &m->xc, es * T * xc));
    DEC_TRY(dalloc(m, &m->scan_y, es * T * sy));
    DEC_TRY(dalloc(m, &m->proj, 4 * T * proj));
    DEC_TRY(dalloc(m, &m->dt_raw, 4 * T * dtr));
    DEC_TRY(dalloc(m, &m->head_gate, 4 * T * gates));
    DEC_TRY(dalloc(m, &m->attn_ctrs, sizeof(int) * attn_counters()));
    DEC_TRY(dalloc(m, &m->dt_op, 2 * T * rp));
    DEC_TRY(dalloc(m, &m->act, es * T * ff));
    if (m->f32) DEC_TRY(dalloc(m, &m->gate32, 2 * 4 * T * ff));
    DEC_TRY(dalloc(m, &m->gathered, 2 * (size_t)m->kv_rows * gat));
    DEC_TRY(dalloc(m, &m->expanded, 2 * (size_t)m->kv_rows * exp_cols));
    m->part_floats = m->f32 ? 0 : part;
    DEC_TRY(dalloc(m, &m->part, 4 * m->part_floats));
    DEC_TRY(dalloc(m, &m->head_in, es * (size_t)m->cap_rows * wp));
    DEC_TRY(dalloc(m, &m->logits, 4 * (size_t)m->cap_rows * m->vp));
    DEC_TRY(dalloc(m, &m->keys, 8 * (size_t)m->cap_rows));
    DEC_TRY(dalloc(m, &m->key_ctrs, 4 * (size_t)m->cap_rows));
    DEC_TRY(dalloc(m, &m->next_dev, 4 * (size_t)m->cap_rows));
    // (partials of a split row-major projection: at most one 128 x 128 tile per SM)
    m->ws_floats = std::max(m->ws_floats, (size_t)sm_count() * 128 * 128);
    m->n_counters = std::max(m->n_counters, sm_count());
    DEC_TRY(dalloc(m, &m->ws, 4 * m->ws_floats));
    DEC_TRY(dalloc(m, &m->counters, 4 * (size_t)m->n_counters));
    std::map<std::pair<int, int>, int> tilings;
    for (const DecLayer& L : m->layers)
        if (L.is_attention()) tilings[L.tiling(false)] = tilings[L.tiling(true)] = 1;
    m->meta_cap = 4 * T + 5 * T + 64;
    const size_t max_chunks = T / REC_CHUNK + c.max_batch;
    if (m->chunk_bytes > 0) {
        DEC_TRY(dalloc(m, &m->chunk_ws, m->chunk_bytes * max_chunks));
        m->meta_cap += 2 * max_chunks + c.max_batch;
    }
    for (auto& t : tilings) m->meta_cap += 2 * (T * t.first.first / t.first.second + T + 1);
    DEC_TRY(dalloc(m, &m->meta, 4 * m->meta_cap));
    JSM_CUDA_CHECK(cudaMallocHost(reinterpret_cast<void**>(&m->h_meta), 4 * m->meta_cap));
    tc_error_word();  // first use allocates the device's error word: here, not inside a captured step
    // bytes of weights one decode step streams (a shared layer streams them again)
    auto pb = [&](const Proj& p) { return (uint64_t)(p.paired ? 2 : 1) * p.N * p.K * es; };
    m->weight_bytes = pb(m->head);
    for (const DecLayer& L : m->layers) {
        m->weight_bytes += pb(L.qd) + pb(L.in) + pb(L.xp) + pb(L.out) + pb(L.gate) + pb(L.up) + pb(L.down);
        if (L.c.mixer == JSM_MIXER_LATENT_ATTENTION) m->weight_bytes += (uint64_t)L.ld.H * (L.ld.dim + L.ld.vdim) * L.ld.rank * es;
        else if (L.c.mixer == JSM_MIXER_SELECTIVE_SCAN) m->weight_bytes += pb(L.dt);
    }
    JSM_CUDA_CHECK(cudaDeviceSynchronize());
    m->ready = true;
    return JSM_OK;
}

static jsm_status check_ready(jsm_decoder* m, const char* who) {
    if (!m) JSM_FAIL(JSM_INVALID_ARG, "%s: null model", who);
    if (!m->ready) JSM_FAIL(JSM_INVALID_ARG, "%s: the model's weights are not finalized (jsm_decoder_finalize)", who);
    return JSM_OK;
}

jsm_status jsm_decoder_seq_open(jsm_decoder* m, int* row) {
    DEC_TRY(check_ready(m, "jsm_decoder_seq_open"));
    if (!row) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_seq_open: null argument");
    if (m->rows.n_active >= m->c.max_batch) JSM_FAIL(JSM_OOM, "jsm_decoder_seq_open: all %d batch rows are in use", m->c.max_batch);
    const int r = m->rows.n_active++;
    m->rows.h_ctx[r] = 0;
    m->slot_of_row[r] = m->free_slots.back();
    m->free_slots.pop_back();
    *row = r;
    return JSM_OK;
}

jsm_status jsm_decoder_seq_retire(jsm_decoder* m, int row, int* moved_from, void* stream) {
    DEC_TRY(check_ready(m, "jsm_decoder_seq_retire"));
    if (row < 0 || row >= m->rows.n_active) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_seq_retire: row %d of %d active", row, m->rows.n_active);
    cudaStream_t st = stream ? as_stream(stream) : m->own_stream;
    m->free_slots.push_back(m->slot_of_row[row]);
    m->slot_of_row[row] = m->slot_of_row[m->rows.n_active - 1];
    return m->rows.retire(row, moved_from, nullptr, st);
}

jsm_status jsm_decoder_step(jsm_decoder* m, int n_entries, const int32_t* rows, const int32_t* counts, const int32_t* h_ids, int n_want,
                            const int32_t* want, int32_t* h_next, float* h_logits, void* stream) {
    DEC_TRY(check_ready(m, "jsm_decoder_step"));
    if (n_entries <= 0) return JSM_OK;
    if (!rows || !counts || !h_ids || (n_want > 0 && !want)) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_step: null argument");
    cudaStream_t st = stream ? as_stream(stream) : m->own_stream;
    std::vector<PassSeg> segs;
    std::vector<char> seen(m->c.max_batch, 0);
    int total = 0;
    for (int e = 0; e < n_entries; ++e) {
        const int r = rows[e];
        if (r < 0 || r >= m->rows.n_active || seen[r]) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_step: row %d (%d active, each at most once)", r, m->rows.n_active);
        if (counts[e] <= 0) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_step: %d tokens for row %d", counts[e], r);
        if (m->rows.h_ctx[r] + counts[e] > m->c.max_context)
            JSM_FAIL(JSM_SHAPE, "context overflow: row %d holds %d tokens and gets %d, the model was created for %d", r, m->rows.h_ctx[r], counts[e], m->c.max_context);
        seen[r] = 1;
        total += counts[e];
    }
    for (int i = 0; i < total; ++i)
        if (h_ids[i] < 0 || h_ids[i] >= m->c.vocab) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_step: token %d outside the vocabulary", h_ids[i]);
    for (int k = 0; k < n_want; ++k)
        if (want[k] < 0 || want[k] >= total) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_step: logits of place %d of %d", want[k], total);
    // passes of at most max_step_tokens tokens
    int used = 0, tok = 0;
    auto flush = [&]() -> jsm_status {
        if (segs.empty()) return JSM_OK;
        std::vector<std::pair<int, int>> w;
        for (int k = 0; k < n_want; ++k)
            for (const PassSeg& s : segs)
                if (want[k] >= s.tok0 && want[k] < s.tok0 + s.len) w.push_back({want[k], k});
        jsm_status s = run_pass(m, segs, h_ids, w, h_next, h_logits, st);
        segs.clear();
        used = 0;
        return s;
    };
    for (int e = 0; e < n_entries; ++e) {
        int left = counts[e], pos = m->rows.h_ctx[rows[e]];
        while (left > 0) {
            if (used == m->c.max_step_tokens) DEC_TRY(flush());
            const int n = std::min(left, m->c.max_step_tokens - used);
            segs.push_back(PassSeg{e, rows[e], tok, n, pos});
            used += n; tok += n; pos += n; left -= n;
            if (left > 0) DEC_TRY(flush());
        }
    }
    return flush();
}

jsm_status jsm_decoder_seq_admit(jsm_decoder* m, const int32_t* h_prompt, int T, int* row_out, int32_t* h_first_token, float* h_logits_last,
                                 void* stream) {
    if (!h_prompt || !row_out) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_seq_admit: null argument");
    if (T <= 0) JSM_FAIL(JSM_SHAPE, "jsm_decoder_seq_admit: %d prompt tokens", T);
    int row = 0;
    DEC_TRY(jsm_decoder_seq_open(m, &row));
    const int32_t r = row, n = T, want = T - 1;
    jsm_status s = jsm_decoder_step(m, 1, &r, &n, h_prompt, 1, &want, h_first_token, h_logits_last, stream);
    if (s != JSM_OK) {  // a refused admission takes nothing
        const std::string why = jsm_last_error();
        jsm_decoder_seq_retire(m, row, nullptr, stream);
        set_error("%s", why.c_str());
        return s;
    }
    *row_out = row;
    return JSM_OK;
}

jsm_status jsm_decoder_step_active(jsm_decoder* m, const int32_t* h_ids, int32_t* h_next, float* h_logits, void* stream) {
    DEC_TRY(check_ready(m, "jsm_decoder_step_active"));
    if (!h_ids || !h_next) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_step_active: null argument");
    const int n = m->rows.n_active;
    std::vector<int32_t> rows(n), ones(n, 1);
    for (int i = 0; i < n; ++i) rows[i] = i;
    return jsm_decoder_step(m, n, rows.data(), ones.data(), h_ids, n, rows.data(), h_next, h_logits, stream);
}

jsm_status jsm_decoder_pool_state(jsm_decoder* m, int* n_active, int* free_pages, int* total_pages) {
    DEC_TRY(check_ready(m, "jsm_decoder_pool_state"));
    if (n_active) *n_active = m->rows.n_active;
    if (free_pages) *free_pages = (int)m->rows.free_pages.size();
    if (total_pages) *total_pages = m->rows.n_pool_pages;
    return JSM_OK;
}

jsm_status jsm_decoder_context(jsm_decoder* m, int row, int* context_len) {
    DEC_TRY(check_ready(m, "jsm_decoder_context"));
    if (row < 0 || row >= m->rows.n_active || !context_len) JSM_FAIL(JSM_INVALID_ARG, "jsm_decoder_context: row %d", row);
    *context_len = m->rows.h_ctx[row];
    return JSM_OK;
}

jsm_status jsm_decoder_set_tap(jsm_decoder* m, float* d_buf) {
    DEC_TRY(check_ready(m, "jsm_decoder_set_tap"));
    m->tap = d_buf;
    return JSM_OK;
}

jsm_status jsm_decoder_step_bytes(jsm_decoder* m, int context_len, uint64_t* weight_bytes, uint64_t* seq_bytes) {
    DEC_TRY(check_ready(m, "jsm_decoder_step_bytes"));
    if (weight_bytes) *weight_bytes = m->weight_bytes;
    if (seq_bytes) {
        const uint64_t es = m->f32 ? 4 : 2;
        *seq_bytes = 0;
        for (const DecLayer& L : m->layers) {
            if (L.c.mixer == JSM_MIXER_LATENT_ATTENTION) *seq_bytes += (uint64_t)std::min(context_len, L.ld.window) * L.ld.cr() * es;
            else if (L.c.mixer == JSM_MIXER_ATTENTION)
                *seq_bytes += (uint64_t)std::min(context_len, L.ad.mask.reach(context_len)) * L.ad.G * (L.ad.ks() + L.ad.vs()) * 64 * es;
            else if (L.is_recurrence())
                *seq_bytes += 2ull * (4ull * L.rd.H * L.rd.kp() * L.rd.vp() + es * (L.rd.taps - 1) * L.rd.conv_cols());
            else *seq_bytes += 2ull * (4ull * L.sd.ip() * L.sd.np() + es * (L.sd.taps - 1) * L.sd.ip());
        }
    }
    return JSM_OK;
}

}  // extern "C"
#undef DEC_TRY
