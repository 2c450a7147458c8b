/*
 * vb_lm.cu - decoder language models: weight loading, slots with caches and states, the step
 * function, greedy generation, and the C ABI (voxtral_b200_lm.h).
 *
 * A step is a fixed sequence of launches per layer:
 *   [loop projection,] in-projection GEMM, mixer kernels, out-projection GEMM, residual + norms,
 *   gate/up GEMM (SwiGLU epilogue), down GEMM, residual + norms
 * or, where one norm feeds mixer and feed-forward,
 *   GEMM of every projection that reads the norm, mixer kernels [, experts], GEMM of the two
 *   out-projections side by side, residual + norm
 * with the GEMMs of vb_tc.cu (split-K partials, summed by the consumer) and, in the 32-bit mode,
 * a plain fp32 GEMM in their place. One-token steps are captured once as a CUDA graph and
 * replayed for every position and slot.
 */
#include "../../include/voxtral_b200_lm.h"
#include "vb_lm_config.h"
#include "vb_lm_kernels.cuh"
#include "vb_safetensors.h"
#include "vb_tc.cuh"
#include "vb_upload.cuh"

#include <math.h>
#include <stdio.h>
#include <stdlib.h>
#include <string.h>

#include <algorithm>
#include <map>
#include <memory>
#include <string>
#include <vector>

namespace vb {

namespace {

thread_local std::string g_error;

int fail(const std::string &what) {
    g_error = what;
    return -1;
}
int cuda_ok(cudaError_t e, const char *what) {
    if (e == cudaSuccess) return 0;
    return fail(std::string(what) + ": " + cudaGetErrorString(e));
}
#define LM_CUDA(call)                                \
    do {                                             \
        if (cuda_ok((call), #call)) return -1;       \
    } while (0)
#define LM_DO(call)                                                                                   \
    do {                                                                                              \
        if (call) return g_error.empty() ? fail(std::string(#call) + " could not be launched") : -1;  \
    } while (0)

int round_up(int v, int to) { return (v + to - 1) / to * to; }

/* ------------------------------------------------------------------ weights */
/* Where tensors come from: a safetensors file, or hashed values of the right shapes. */
struct Source {
    const SafeTensors *file = nullptr;
    unsigned seed = 0;
};

struct Linear {
    uint16_t *W = nullptr;      /* tile-contiguous (tensor cores) or row-major [N][Kp] (fp32) */
    TcWeight tc;
    int N = 0, K = 0, Kp = 0;   /* N padded to a multiple of 4, K padded to whole 64-column blocks */
    bool swiglu = false;
    /* rows from act_n0 on are a feed-forward's: their results, max(., 0)^2, belong in columns act_col... of act_acts
     * (written by the GEMM itself for many rows, by the mixer's preparation otherwise); 0: none */
    int act_n0 = 0, act_col = 0;
    struct Acts *act_acts = nullptr;
};

/* Rows that feed a GEMM, as BF16 terms or fp32; columns [K, Kp) stay zero. */
struct Acts {
    uint16_t *terms = nullptr;
    float *rows = nullptr;
    int K = 0, Kp = 0;
    std::map<int, TcActs> maps;   /* by padded row count */
};

struct Mixer {
    Linear in, out;
    Acts *acts = nullptr;         /* rows that `out` reads */
    /* attention */
    float *q_gain = nullptr, *k_gain = nullptr, *freq = nullptr;
    float mag = 1.0f;
    /* delta rule */
    float *conv = nullptr, *decay = nullptr, *dt_bias = nullptr, *norm = nullptr;
    /* latent attention */
    Linear uq, ukv;               /* query out of its latent; keys and values out of the cached one */
    Acts *uq_acts = nullptr, *kv_acts = nullptr;
    float *c_gain = nullptr;
    int col_c = 0, col_g = 0, col_router = 0;   /* columns of the in-projection (query latent: 0) */
};

struct Layer {
    float *norm1 = nullptr, *norm1b = nullptr, *norm2 = nullptr, *norm2b = nullptr;
    Mixer mix;
    Linear up, down;              /* gate and up rows interleaved; a mixture's experts one below the other */
    Acts *ff_acts = nullptr;
    int expert_rows = 0, expert_rows_down = 0;   /* rows from one expert's matrix to the next */
};

/* Cache or state of one layer run inside a slot's slab: offsets in floats. */
struct RunState {
    size_t a = 0, b = 0;          /* attention: K, V; delta: S, convolution memory; latent: the cache (a) */
    LmRing ring = {0, 1};
};

enum Variant { STEP_SILENT = 0, STEP_LOGITS = 1, STEP_GREEDY = 2, kVariants = 3 };
constexpr int kHeadRows = 64;     /* rows that go through the head at once */
constexpr int kLogCap = 1 << 16;  /* generated tokens kept on the device */

} // namespace

} // namespace vb

using namespace vb;

struct vb200_lm {
    LmConfig cfg;
    std::vector<LmConfig::Run> runs;
    int dtype = VB200_LM_BF16, max_seqs = 1, max_tokens = 0, block = 0, n_sm = 0;
    bool f32() const { return dtype == VB200_LM_F32; }

    cudaStream_t st = nullptr;
    std::vector<void *> allocs;
    std::vector<std::unique_ptr<Acts>> acts;
    std::vector<Layer> layers;
    uint16_t *embed = nullptr;
    float *final_norm = nullptr;
    Linear loop_in, head;
    Acts *x_acts = nullptr, *loop_acts = nullptr;
    size_t weight_bytes = 0;

    /* slots */
    std::vector<RunState> states;
    float *slabs = nullptr;
    size_t slab = 0;
    struct Seq { bool open = false; int length = 0; };
    std::vector<Seq> seqs;

    /* activations */
    float *x = nullptr, *part_in = nullptr, *part_out = nullptr, *part_head = nullptr, *logits = nullptr;
    float *q = nullptr, *k = nullptr, *v = nullptr, *o = nullptr, *beta = nullptr, *decays = nullptr, *gram = nullptr;
    float *scratch = nullptr, *tap = nullptr;
    unsigned *tickets = nullptr;
    int *status = nullptr, *log = nullptr, *zero = nullptr;
    /* latent attention */
    float *part_q = nullptr, *gate = nullptr, *cs = nullptr, *ql = nullptr;
    uint16_t *wide = nullptr;            /* keys and values of a stretch, written out */
    struct { const Acts *acts = nullptr; size_t cache = 0; int first = 0, n = 0; } gathered;   /* what kv_acts hold within a step */
    int pos_now = 0;                     /* position of the first row of the launch sequence being enqueued */
    /* mixture of experts */
    Acts *sorted_acts = nullptr;
    std::map<int, Acts *> expert_acts;   /* by expert size */
    int sorted_rows = 0, y_ld = 0;
    float *expert_y = nullptr, *few_act = nullptr, *route_weight = nullptr;
    int *route = nullptr, *route_at = nullptr;
    int4 *route_table = nullptr;
    bool tap_on = false;
    int tap_rows = 0;

    /* one host block -> device block per launch sequence: LmDyn, tokens, wanted rows */
    int *d_in = nullptr, *h_in[2] = {};
    cudaEvent_t in_free[2] = {};
    bool in_busy[2] = {};
    int in_next = 0;
    LmDyn *dyn() const { return (LmDyn *)d_in; }
    int *tokens() const { return d_in + 4; }
    int *wanted() const { return d_in + 4 + block; }

    cudaGraphExec_t exec[kVariants] = {};
    int direct_calls[kVariants] = {};
    cudaEvent_t ev[3] = {};
    bool timed = false;

    ~vb200_lm();
    int init(const Source &src, const vb200_lm_options_t *opt);
    int enqueue(int M, int n_want, float *logits_out, bool greedy);
    int launch(int M, int n_want, float *logits_out, bool greedy);
    int feed(int seq, const int *tok, int M, const int *want, int n_want);
    int finish();

private:
    template <typename T> int alloc(T **p, size_t n, bool clear = false);
    int tensor(const Source &s, const std::string &name, std::vector<int64_t> shape, uint16_t *dst, Stager *stage);
    int host_tensor(const Source &s, const std::string &name, std::vector<int64_t> shape, std::vector<float> *out);
    int upload(const std::vector<float> &h, float **d);
    int gain(const Source &s, const std::string &name, int n, float **d);
    struct Piece { std::string name; int rows, cols, row0, step, col0 = 0; };
    int linear(const Source &s, const std::vector<Piece> &pieces, int N, int K, bool swiglu, Linear *l);
    int make_acts(int K, Acts **out, int rows = 0);
    int load_mixer(const Source &s, const LmMixer &m, const std::string &mp, Mixer *x);
    int load_latent(const Source &s, const LmLayer &spec, const std::string &mp, Layer *l);
    int load_experts(const Source &s, const LmMlp &m, const std::string &fp, Layer *l);
    int load(const Source &s);
    int make_state();
    int make_buffers();

    int splits_of(const Linear &l, int M) const;
    bool fused_act(const Linear &l, int M) const { return !f32() && l.act_n0 > 0 && M > 256; }
    size_t part_floats(const Linear &l, int max_rows) const;
    TcActs *map_of(Acts *a, int M);
    LmSink sink(Acts *a, int M);
    int gemm(const Linear &l, Acts *in, int M, float *part, Acts *swiglu_out, LmPart *out);
    int mixer(const Layer &l, const LmLayer &spec, const RunState &s, int M);
    int latent(const Layer &l, const LmLayer &spec, const RunState &s, int M);
    int latent_wide(const Layer &l, const LmMixer &m, const LmLatent &a, const RunState &s, int M);
    int experts(const Layer &l, const LmMlp &m, int M, LmMix *mix);
    bool latent_split(const LmMixer &m) const { return !f32() && lm_latent_split_ok(m.kv_rank, m.rot_dim); }
    int wide_rows(const LmMixer &m) const {
        return m.mask.window > 0 ? (int)std::min((long long)max_tokens, (long long)m.mask.window - 1 + block) : max_tokens;
    }
    /* prompts write keys and values out where the sizes allow it; rows that never do */
    bool latent_wide_ok(const LmMixer &m) const {
        return latent_split(m) && lm_attn_wide_ok(m.dim, m.rot_dim, m.vdim) && wide_rows(m) <= kTcMaxRows;
    }
    int absorb_rows(const LmMixer &m) const { return latent_wide_ok(m) ? std::min(block, kLmLatentRows) : block; }

    Stager stage_;
    uint16_t *tmp_ = nullptr;     /* upload staging on the device */
    size_t tmp_cap_ = 0;
};

/* ------------------------------------------------------------------ memory */
template <typename T> int vb200_lm::alloc(T **p, size_t n, bool clear) {
    void *q = nullptr;
    const size_t bytes = std::max<size_t>(n * sizeof(T), 16);
    if (cudaMalloc(&q, bytes) != cudaSuccess) {
        cudaGetLastError();
        return fail("out of device memory (" + std::to_string(bytes) + " bytes)");
    }
    allocs.push_back(q);
    if (clear) LM_CUDA(cudaMemsetAsync(q, 0, bytes, st));
    *p = (T *)q;
    return 0;
}

vb200_lm::~vb200_lm() {
    if (st) cudaStreamSynchronize(st);
    for (int i = 0; i < kVariants; i++)
        if (exec[i]) cudaGraphExecDestroy(exec[i]);
    stage_.close();
    for (int i = 0; i < 2; i++) {
        if (h_in[i]) cudaFreeHost(h_in[i]);
        if (in_free[i]) cudaEventDestroy(in_free[i]);
    }
    for (cudaEvent_t e : ev)
        if (e) cudaEventDestroy(e);
    for (void *p : allocs) cudaFree(p);
    if (st) cudaStreamDestroy(st);
    cudaGetLastError();
}

/* ------------------------------------------------------------------ loading */
static float hashed(unsigned &h) {   /* about N(0, 1) */
    float s = 0.0f;
    for (int i = 0; i < 4; i++) {
        h = h * 1664525u + 1013904223u;
        s += (float)(h >> 8) / 16777216.0f - 0.5f;
    }
    return s * 1.7320508f;
}
static unsigned hash_name(const std::string &n, unsigned seed) {
    unsigned h = 2166136261u ^ seed;
    for (char c : n) h = (h ^ (unsigned char)c) * 16777619u;
    return h;
}

static std::string shape_text(const std::vector<int64_t> &s) {
    std::string t = "[";
    for (size_t i = 0; i < s.size(); i++) t += (i ? ", " : "") + std::to_string(s[i]);
    return t + "]";
}

static const Tensor *checked(const SafeTensors *f, const std::string &name, const std::vector<int64_t> &shape) {
    const Tensor *t = f->find(name);
    if (!t) { fail("model.safetensors has no tensor '" + name + "'"); return nullptr; }
    if (t->dtype != "BF16") { fail("tensor '" + name + "' is " + t->dtype + ", expected BF16"); return nullptr; }
    if (t->shape != shape) {
        fail("tensor '" + name + "' is " + shape_text(t->shape) + ", the configuration asks for " + shape_text(shape));
        return nullptr;
    }
    return t;
}

/* A BF16 tensor to device memory as it lies in the file. */
int vb200_lm::tensor(const Source &s, const std::string &name, std::vector<int64_t> shape, uint16_t *dst, Stager *stage) {
    size_t n = 1;
    for (int64_t d : shape) n *= (size_t)d;
    if (!s.file) return lm_fill_random(dst, n, hash_name(name, s.seed), 0.0f, 0.02f, st) ? fail("random fill failed") : 0;
    const Tensor *t = checked(s.file, name, shape);
    if (!t) return -1;
    return stage->copy(dst, t->data, t->bytes, st) ? fail("upload of '" + name + "' failed") : 0;
}

/* A small BF16 tensor as host floats. */
int vb200_lm::host_tensor(const Source &s, const std::string &name, std::vector<int64_t> shape, std::vector<float> *out) {
    size_t n = 1;
    for (int64_t d : shape) n *= (size_t)d;
    out->resize(n);
    if (!s.file) {
        unsigned h = hash_name(name, s.seed);
        const bool is_gain = name.find("norm") != std::string::npos, is_decay = name.find("A_log") != std::string::npos;
        for (float &v : *out) v = is_gain ? 1.0f + 0.02f * hashed(h) : is_decay ? 0.5f * hashed(h) : 0.3f * hashed(h);
        return 0;
    }
    const Tensor *t = checked(s.file, name, shape);
    if (!t) return -1;
    for (size_t i = 0; i < n; i++) {
        uint16_t b;
        memcpy(&b, (const char *)t->data + 2 * i, 2);
        const uint32_t u = (uint32_t)b << 16;
        memcpy(&(*out)[i], &u, 4);
    }
    return 0;
}

int vb200_lm::upload(const std::vector<float> &h, float **d) {
    if (alloc(d, h.size())) return -1;
    LM_CUDA(cudaMemcpyAsync(*d, h.data(), h.size() * sizeof(float), cudaMemcpyHostToDevice, st));
    LM_CUDA(cudaStreamSynchronize(st));
    return 0;
}

int vb200_lm::gain(const Source &s, const std::string &name, int n, float **d) {
    std::vector<float> h;
    return host_tensor(s, name, {n}, &h) || upload(h, d) ? -1 : 0;
}

/* One GEMM's weight matrix out of several tensors: row r of a piece becomes row row0 + r * step, from column col0 on. */
int vb200_lm::linear(const Source &s, const std::vector<Piece> &pieces, int N, int K, bool swiglu, Linear *l) {
    l->N = round_up(N, 4); l->K = K; l->Kp = round_up(K, kTcBlockK); l->swiglu = swiglu;
    const size_t elems = (size_t)l->N * l->Kp;
    uint16_t *rows = nullptr;
    if (cudaMalloc(&rows, elems * 2) != cudaSuccess) {
        cudaGetLastError();
        return fail("out of device memory for a weight matrix");
    }
    int rc = cuda_ok(cudaMemsetAsync(rows, 0, elems * 2, st), "memset");
    for (const Piece &p : pieces) {
        if (rc) break;
        const size_t n = (size_t)p.rows * p.cols;
        if (n > tmp_cap_) {
            cudaStreamSynchronize(st);
            cudaFree(tmp_);
            tmp_cap_ = 0;
            rc = cuda_ok(cudaMalloc(&tmp_, n * 2), "staging buffer");
            if (rc) { tmp_ = nullptr; break; }
            tmp_cap_ = n;
        }
        rc = tensor(s, p.name, {p.rows, p.cols}, tmp_, &stage_);
        if (!rc && lm_pack_rows(rows, l->Kp, p.row0, p.step, p.col0, tmp_, p.rows, p.cols, st)) rc = fail("weight packing failed");
    }
    if (!rc && !f32()) {
        uint16_t *tiled = nullptr;
        rc = alloc(&tiled, tc_tiled_bytes(l->N, l->Kp) / 2);
        if (!rc && tc_weight_tiled(&l->tc, rows, l->N, l->Kp, tiled, st)) rc = fail("tensor map of a weight matrix could not be made");
        if (!rc) rc = cuda_ok(cudaStreamSynchronize(st), "weight upload");
        l->W = tiled;
        cudaFree(rows);
        weight_bytes += tc_tiled_bytes(l->N, l->Kp);
    } else {
        allocs.push_back(rows);
        l->W = rows;
        weight_bytes += elems * 2;
    }
    return rc;
}

/* rows: 0 for as many as a block or the head has; otherwise that many, in two terms (row-block GEMMs only). */
int vb200_lm::make_acts(int K, Acts **out, int rows) {
    acts.emplace_back(new Acts());
    Acts *a = acts.back().get();
    a->K = K;
    a->Kp = round_up(K, kTcBlockK);
    *out = a;
    const int n = rows > 0 ? rows : std::max(block, kHeadRows);
    if (f32()) return alloc(&a->rows, (size_t)n * a->Kp, true);
    if (rows > 0) return alloc(&a->terms, (size_t)2 * round_up(std::max(rows, 256), 128) * a->Kp, true);
    return alloc(&a->terms, tc_acts_bytes(std::max(tc_rows_pad_any(n), 64), a->Kp) / 2, true);
}

/* In-projection of an attention or a delta-rule mixer: all of its projections below one another. */
int vb200_lm::load_mixer(const Source &s, const LmMixer &m, const std::string &mp, Mixer *x) {
    const int W = cfg.width;
    const int nq = m.kind == LM_MIXER_DELTA ? m.kv_heads * m.dim : m.heads * m.dim, nk = m.kv_heads * m.dim;
    const int nv = (m.kind == LM_MIXER_DELTA ? m.heads : m.kv_heads) * m.vdim, no = m.heads * m.vdim;
    std::vector<Piece> in = {{mp + "q", nq, W, 0, 1}, {mp + "k", nk, W, nq, 1}, {mp + "v", nv, W, nq + nk, 1}};
    int N = nq + nk + nv;
    if (m.kind == LM_MIXER_DELTA) {
        in.push_back({mp + "g", no, W, N, 1});
        in.push_back({mp + "b", m.heads, W, N + no, 1});
        in.push_back({mp + "a", m.heads, W, N + no + m.heads, 1});
        N += no + 2 * m.heads;
        std::vector<float> conv, part, alog, v;
        const struct { const char *n; int ch; } cs[3] = {{"q.conv", nq}, {"k.conv", nk}, {"v.conv", nv}};
        for (const auto &c : cs) {
            if (host_tensor(s, mp + c.n, {c.ch, m.taps}, &part)) return -1;
            conv.insert(conv.end(), part.begin(), part.end());
        }
        if (host_tensor(s, mp + "A_log", {m.heads}, &alog)) return -1;
        for (float &y : alog) y = (float)exp((double)y);
        if (upload(conv, &x->conv) || upload(alog, &x->decay) || gain(s, mp + "dt_bias", m.heads, &x->dt_bias) ||
            gain(s, mp + "norm", m.vdim, &x->norm))
            return -1;
    } else {
        if (gain(s, mp + "q.norm", nq, &x->q_gain) || gain(s, mp + "k.norm", nk, &x->k_gain)) return -1;
    }
    return linear(s, in, N, W, false, &x->in) || linear(s, {{mp + "o", W, no, 0, 1}}, W, no, false, &x->out) ? -1 : 0;
}

/* In-projection: [query latent | latent and key part | gates | router | feed-forward], every part on a multiple of four
 * columns, the feed-forward on whole tiles. Out-projection: [heads | feed-forward] side by side. */
int vb200_lm::load_latent(const Source &s, const LmLayer &spec, const std::string &mp, Layer *l) {
    const LmMixer &m = spec.mixer;
    const int W = cfg.width, no = m.heads * m.vdim;
    const bool parallel = cfg.block == LM_BLOCK_PARALLEL, own = m.kv_from < 0;
    const std::string fp = mp.substr(0, mp.size() - 4) + "mlp.";
    Mixer &x = l->mix;
    std::vector<Piece> in = {{mp + "dq", m.q_rank, W, 0, 1}};
    int N = round_up(m.q_rank, 4);
    x.col_c = N;
    if (own) {
        in.push_back({mp + "dkv", m.kv_rank + m.rot_dim, W, N, 1});
        N = round_up(N + m.kv_rank + m.rot_dim, 4);
    }
    x.col_g = N;
    in.push_back({mp + "g", m.heads, W, N, 1});
    N = round_up(N + m.heads, 4);
    x.col_router = N;
    if (parallel && spec.mlp.experts > 0) {
        in.push_back({fp + "router", spec.mlp.experts, W, N, 1});
        N += spec.mlp.experts;
    }
    const int ff = parallel && spec.mlp.experts == 0 ? spec.mlp.ff : 0, ff_out = round_up(no, kTcBlockK);
    std::vector<Piece> out = {{mp + "o", W, no, 0, 1}};
    if (ff > 0) {
        x.in.act_n0 = round_up(N, kTcTileN);
        x.in.act_col = ff_out;
        in.push_back({fp + "up", ff, W, x.in.act_n0, 1});
        out.push_back({fp + "down", W, ff, 0, 1, ff_out});
        N = x.in.act_n0 + ff;
    }
    if (linear(s, in, N, W, false, &x.in) || linear(s, out, W, ff > 0 ? ff_out + ff : no, false, &x.out) ||
        linear(s, {{mp + "uq", m.heads * (m.dim + m.rot_dim), m.q_rank, 0, 1}}, m.heads * (m.dim + m.rot_dim), m.q_rank, false, &x.uq) ||
        linear(s, {{mp + "uk", m.heads * m.dim, m.kv_rank, 0, 1}, {mp + "uv", no, m.kv_rank, m.heads * m.dim, 1}}, m.heads * (m.dim + m.vdim),
               m.kv_rank, false, &x.ukv))
        return -1;
    return gain(s, mp + "dq.norm", m.q_rank, &x.q_gain) || (own && gain(s, mp + "dkv.norm", m.kv_rank, &x.c_gain)) ? -1 : 0;
}

int vb200_lm::load_experts(const Source &s, const LmMlp &m, const std::string &fp, Layer *l) {
    const int W = cfg.width;
    l->expert_rows = round_up(m.ff, kTcTileN);
    l->expert_rows_down = round_up(W, kTcTileN);
    std::vector<Piece> up, down;
    for (int e = 0; e < m.experts; e++) {
        const std::string ep = fp + "e" + std::to_string(e) + ".";
        up.push_back({ep + "up", m.ff, W, e * l->expert_rows, 1});
        down.push_back({ep + "down", W, m.ff, e * l->expert_rows_down, 1});
    }
    return linear(s, up, m.experts * l->expert_rows, W, false, &l->up) ||
                   linear(s, down, m.experts * l->expert_rows_down, m.ff, false, &l->down)
               ? -1
               : 0;
}

int vb200_lm::load(const Source &s) {
    const int W = cfg.width;
    stage_.open();
    if (alloc(&embed, (size_t)cfg.vocab * W) || tensor(s, "embed", {cfg.vocab, W}, embed, &stage_)) return -1;
    weight_bytes += (size_t)cfg.vocab * W * 2;
    if (make_acts(W, &x_acts)) return -1;
    if (cfg.loop_times > 0) {
        if (linear(s, {{"loop.in", W, 2 * W, 0, 1}}, W, 2 * W, false, &loop_in) || make_acts(2 * W, &loop_acts)) return -1;
    }
    std::map<std::pair<int, int>, Acts *> mix_acts;   /* layers of equal sizes share the rows between two GEMMs */
    std::map<int, Acts *> ff_acts, latent_acts;
    layers.resize(cfg.layers.size());
    for (size_t i = 0; i < layers.size(); i++) {
        const LmLayer &spec = cfg.layers[i];
        const LmMixer &m = spec.mixer;
        Layer &l = layers[i];
        const std::string p = "l" + std::to_string(i) + ".", mp = p + "mix.";
        const bool parallel = cfg.block == LM_BLOCK_PARALLEL;
        if (gain(s, p + "norm1", W, &l.norm1) || (!parallel && gain(s, p + "norm1b", W, &l.norm1b))) return -1;
        if (m.rope.dims > 0) {
            const std::vector<double> f = m.rope.frequencies();
            std::vector<float> hl(2 * f.size());
            for (size_t j = 0; j < f.size(); j++) {
                hl[j] = (float)f[j];
                hl[f.size() + j] = (float)(f[j] - (double)hl[j]);
            }
            if (upload(hl, &l.mix.freq)) return -1;
            l.mix.mag = (float)m.rope.magnitude();
        }
        if (m.kind == LM_MIXER_LATENT ? load_latent(s, spec, mp, &l) : load_mixer(s, m, mp, &l.mix)) return -1;
        const int no = m.heads * m.vdim, ff_out = parallel && spec.mlp.experts == 0 ? spec.mlp.ff : 0;
        Acts *&ma = mix_acts[{no, ff_out}];
        if (!ma && make_acts(l.mix.out.K, &ma)) return -1;
        l.mix.acts = ma;
        if (l.mix.in.act_n0 > 0) l.mix.in.act_acts = ma;
        if (m.kind == LM_MIXER_LATENT) {
            Acts *&qa = latent_acts[m.q_rank];
            if (!qa && make_acts(m.q_rank, &qa)) return -1;
            l.mix.uq_acts = qa;
        }
        const std::string fp = p + "mlp.";
        const int ff = spec.mlp.ff;
        if (spec.mlp.experts > 0) {
            if (load_experts(s, spec.mlp, fp, &l)) return -1;
        } else if (spec.mlp.kind == LM_MLP_SWIGLU) {
            const int ffp = round_up(ff, kTcBlockK);   /* zero rows beyond ff give zero columns */
            if (gain(s, p + "norm2", W, &l.norm2) || gain(s, p + "norm2b", W, &l.norm2b)) return -1;
            if (linear(s, {{fp + "gate", ff, W, 0, 2}, {fp + "up", ff, W, 1, 2}}, 2 * ffp, W, true, &l.up) ||
                linear(s, {{fp + "down", W, ff, 0, 1}}, W, ff, false, &l.down))
                return -1;
            if (!ff_acts[ff] && make_acts(ff, &ff_acts[ff])) return -1;
            l.ff_acts = ff_acts[ff];
        }
    }
    if (gain(s, "final.norm", W, &final_norm) || linear(s, {{"head", cfg.vocab, W, 0, 1}}, cfg.vocab, W, false, &head)) return -1;
    LM_CUDA(cudaStreamSynchronize(st));
    stage_.close();
    cudaFree(tmp_);
    tmp_ = nullptr;
    tmp_cap_ = 0;
    return 0;
}

/* ------------------------------------------------------------------ slots */
int vb200_lm::make_state() {
    size_t at = 0;
    auto take = [&](size_t n) {
        const size_t o = at;
        at += (n + 63) / 64 * 64;
        return o;
    };
    for (const auto &r : runs) {
        const LmMixer &m = cfg.layers[r.layer].mixer;
        RunState s;
        if (m.kv_from >= 0) {             /* another layer's cache (no loop in such a design: run = layer) */
            states.push_back(states[m.kv_from]);
            continue;
        }
        if (m.kind == LM_MIXER_DELTA) {
            s.a = take((size_t)m.heads * m.dim * m.vdim);
            s.b = take((size_t)m.taps * lm_delta_channels(m.heads, m.kv_heads, m.dim, m.vdim));
        } else {
            /* a block's keys are appended before its first row looks back a whole window */
            const int window = cfg.cache_window(r.layer);
            long long keep = window > 0 ? std::min(m.mask.keep_first, max_tokens) : 0;
            long long ring = window > 0 ? (long long)window - 1 + block : max_tokens;
            ring = std::max(1LL, std::min(ring, (long long)max_tokens - keep));
            s.ring.keep = (int)keep;
            s.ring.ring = (int)ring;
            if (m.kind == LM_MIXER_LATENT) {
                s.a = take((size_t)ring * (m.kv_rank + m.rot_dim));
            } else {
                s.a = take((size_t)(keep + ring) * m.kv_heads * m.dim);
                s.b = take((size_t)(keep + ring) * m.kv_heads * m.vdim);
            }
        }
        states.push_back(s);
    }
    slab = at;
    seqs.resize(max_seqs);
    return alloc(&slabs, slab * max_seqs, true);
}

/* ------------------------------------------------------------------ activations */
int vb200_lm::splits_of(const Linear &l, int M) const {
    if (f32() || l.swiglu || fused_act(l, M)) return 1;
    if (M <= 64) return tc_pick_splits(l.N, l.Kp, n_sm);
    /* row-block kernel: a CTA per pair of weight tiles and 128 rows */
    const int tiles = (l.N + kTcTileN - 1) / kTcTileN, ctas = (tiles + 1) / 2 * ((M + 127) / 128);
    return std::max(1, std::min({n_sm / ctas, kTcMaxSplits, l.Kp / kTcBlockK}));
}

size_t vb200_lm::part_floats(const Linear &l, int max_rows) const {
    if (l.swiglu || l.N == 0) return 0;
    size_t n = 0;
    for (int M = 1; M <= max_rows; M++) n = std::max(n, (size_t)splits_of(l, M) * M * (fused_act(l, M) ? l.act_n0 : l.N));
    return n;
}

int vb200_lm::make_buffers() {
    const int W = cfg.width;
    size_t in = 0, out = part_floats(loop_in, block), qn = 0, kn = 0, vn = 0, hn = 0, on = 0, gn = 0, scr = 0;
    size_t pq = 0, gaten = 0, csn = 0, qln = 0, widen = 0, topn = 0, fewn = 0, tablen = 0;
    std::map<int, int> kv_rows;
    int tick = 1;
    for (size_t i = 0; i < layers.size(); i++) {
        const LmMixer &m = cfg.layers[i].mixer;
        in = std::max(in, part_floats(layers[i].mix.in, block));
        out = std::max({out, part_floats(layers[i].mix.out, block), layers[i].ff_acts ? part_floats(layers[i].down, block) : 0});
        const LmMlp &mlp = cfg.layers[i].mlp;
        if (mlp.experts > 0) {
            topn = std::max(topn, (size_t)mlp.top);
            fewn = std::max(fewn, (size_t)mlp.top * round_up(mlp.ff, kTcBlockK));
            tablen = std::max(tablen, (size_t)lm_moe_blocks(block, mlp.experts, mlp.top));
        }
        if (m.kind == LM_MIXER_DELTA) {
            qn = std::max(qn, (size_t)m.kv_heads * m.dim);
            kn = std::max(kn, (size_t)m.kv_heads * m.dim);
            vn = std::max(vn, (size_t)m.heads * m.vdim);
            on = std::max(on, (size_t)m.heads * m.vdim);
            hn = std::max(hn, (size_t)m.heads);
            gn = std::max(gn, (size_t)m.kv_heads);
        } else if (m.kind == LM_MIXER_LATENT) {
            const int rows = absorb_rows(m);
            pq = std::max(pq, part_floats(layers[i].mix.uq, block));
            gaten = std::max(gaten, (size_t)m.heads);
            csn = std::max(csn, (size_t)m.rope.dims);
            qln = std::max(qln, (size_t)rows * m.heads * (m.kv_rank + m.rot_dim));
            scr = std::max(scr, lm_latent_scratch_floats(rows, m.heads, m.kv_rank));
            if (latent_wide_ok(m)) {
                kv_rows[m.kv_rank] = std::max(kv_rows[m.kv_rank], wide_rows(m));
                widen = std::max(widen, (size_t)2 * round_up(std::max(wide_rows(m), 256), 128) * layers[i].mix.ukv.N);
            }
        } else {
            qn = std::max(qn, (size_t)m.heads * m.dim);
            scr = std::max(scr, lm_attn_scratch_floats(m.heads, m.kv_heads, m.vdim));
            tick = std::max(tick, lm_attn_ticket_count(m.heads, m.kv_heads));
        }
    }
    const size_t B = block;
    std::map<int, Acts *> kv_acts;
    for (const auto &k : kv_rows)
        if (make_acts(k.first, &kv_acts[k.first], k.second)) return -1;
    for (size_t i = 0; i < layers.size(); i++) {
        auto it = kv_acts.find(cfg.layers[i].mixer.kv_rank);
        if (it != kv_acts.end()) layers[i].mix.kv_acts = it->second;
    }
    if (tablen > 0) {
        sorted_rows = (int)tablen * 128;
        y_ld = round_up(W, 4);
        if (make_acts(W, &sorted_acts, sorted_rows) || alloc(&expert_y, (size_t)sorted_rows * y_ld)) return -1;
        for (const LmLayer &l : cfg.layers)
            if (l.mlp.experts > 0 && !expert_acts[l.mlp.ff] && make_acts(l.mlp.ff, &expert_acts[l.mlp.ff], sorted_rows)) return -1;
    }
    if (alloc(&part_q, pq) || alloc(&gate, B * gaten) || alloc(&cs, B * csn) || alloc(&ql, qln) || alloc(&wide, widen) ||
        alloc(&route, B * topn, true) || alloc(&route_at, B * topn, true) || alloc(&route_weight, B * topn) || alloc(&route_table, tablen) ||
        alloc(&few_act, kLmMoeRows * fewn))
        return -1;
    if (alloc(&x, B * W) || alloc(&part_in, in) || alloc(&part_out, out) || alloc(&part_head, part_floats(head, kHeadRows)) ||
        alloc(&logits, (size_t)kHeadRows * head.N) || alloc(&q, B * qn) || alloc(&k, B * kn) || alloc(&v, B * vn) || alloc(&o, B * on) ||
        alloc(&beta, B * hn) || alloc(&decays, B * hn) ||
        alloc(&gram, (B + kLmDeltaRows) / kLmDeltaGroup * gn * 2 * kLmDeltaGroup * kLmDeltaGroup) || alloc(&scratch, scr) || alloc(&tickets, (size_t)tick, true) ||
        alloc(&status, 4, true) || alloc(&log, kLogCap, true) || alloc(&zero, 4, true) || alloc(&d_in, 4 + 2 * B, true))
        return -1;
    for (int i = 0; i < 2; i++) {
        LM_CUDA(cudaHostAlloc(&h_in[i], sizeof(int) * (4 + 2 * B), cudaHostAllocDefault));
        LM_CUDA(cudaEventCreateWithFlags(&in_free[i], cudaEventDisableTiming));
    }
    for (cudaEvent_t &e : ev) LM_CUDA(cudaEventCreate(&e));
    LM_CUDA(cudaStreamSynchronize(st));
    return 0;
}

/* What the kernels can run, beyond what the configuration reader checks. */
static int check_sizes(const LmConfig &cfg) {
    if (cfg.width > 16384) return fail("width above 16384");
    for (size_t i = 0; i < cfg.layers.size(); i++) {
        const LmMixer &m = cfg.layers[i].mixer;
        const std::string where = "layers[" + std::to_string(i) + "]: ";
        if (m.kind == LM_MIXER_DELTA && !lm_delta_supported(m.dim, m.vdim)) return fail(where + "delta head size above 256");
        if (m.kind == LM_MIXER_LATENT) {
            if (!lm_latent_supported(m.q_rank, m.kv_rank, m.rot_dim) || m.dim > 1024 || m.q_rank > 16384) return fail(where + "latent sizes are too large");
            if (m.mask.keep_first > 0) return fail(where + "a latent attention keeps no first tokens");
            if ((long long)m.heads * (m.dim + std::max(m.rot_dim, m.vdim)) > (1 << 20)) return fail(where + "heads * dim is too large");
        }
        const LmMlp &mlp = cfg.layers[i].mlp;
        if (mlp.experts > kLmMoeExperts) return fail(where + "more experts than " + std::to_string(kLmMoeExperts));
        if (mlp.kind != LM_MLP_NONE && (cfg.block == LM_BLOCK_PARALLEL ? m.kind != LM_MIXER_LATENT || mlp.kind != LM_MLP_RELU2
                                                                      : mlp.kind != LM_MLP_SWIGLU || mlp.experts > 0))
            return fail(where + "this feed-forward is not built for this kind of layer");
        if (m.kind == LM_MIXER_ATTENTION && (m.dim > 256 || m.vdim > 256)) return fail(where + "attention head size above 256");
        if ((m.kind != LM_MIXER_LATENT && (long long)m.heads * m.dim > 40000) || (long long)m.heads * m.vdim > (1 << 20)) return fail(where + "heads * dim is too large");
    }
    return 0;
}

int vb200_lm::init(const Source &src, const vb200_lm_options_t *opt) {
    dtype = opt ? opt->dtype : VB200_LM_BF16;
    if (dtype != VB200_LM_BF16 && dtype != VB200_LM_F32) return fail("unknown dtype");
    max_seqs = opt && opt->max_seqs > 0 ? opt->max_seqs : 1;
    max_tokens = opt && opt->max_tokens > 0 ? opt->max_tokens : 8192;
    block = opt && opt->block_rows > 0 ? opt->block_rows : (f32() ? 512 : 2048);
    block = std::min({block, max_tokens, kTcMaxRows / 2});
    if (check_sizes(cfg)) return -1;
    runs = cfg.runs();
    int count = 0, major = 0;
    LM_CUDA(cudaGetDeviceCount(&count));
    const char *env = getenv("VB200_DEVICE");
    int dev = env ? atoi(env) : 0;
    if (dev < 0 || dev >= count) dev = 0;
    LM_CUDA(cudaSetDevice(dev));
    LM_CUDA(cudaDeviceGetAttribute(&major, cudaDevAttrComputeCapabilityMajor, dev));
    LM_CUDA(cudaDeviceGetAttribute(&n_sm, cudaDevAttrMultiProcessorCount, dev));
    if (major != 10) return fail("an sm_100 GPU is required");
    if (tc_init()) return fail("tensor maps are not available on this driver");
    LM_CUDA(cudaStreamCreateWithFlags(&st, cudaStreamNonBlocking));
    return load(src) || make_state() || make_buffers() ? -1 : 0;
}

/* ------------------------------------------------------------------ the step */
TcActs *vb200_lm::map_of(Acts *a, int M) {
    const int rp = M <= 256 ? tc_rows_pad_frame(M) : tc_rows_pad_any(M);
    auto it = a->maps.find(rp);
    if (it == a->maps.end()) {
        TcActs t;
        if (tc_acts(&t, a->terms, rp, a->Kp)) return nullptr;
        it = a->maps.emplace(rp, t).first;
    }
    return &it->second;
}

LmSink vb200_lm::sink(Acts *a, int M) {
    LmSink s = {};
    s.ld = a->Kp;
    if (f32()) {
        s.rows = a->rows;
    } else {
        s.terms = a->terms;
        s.rows_pad = M <= 256 ? tc_rows_pad_frame(M) : tc_rows_pad_any(M);
        s.n_terms = M <= 64 ? 3 : 2;      /* the row-block kernel multiplies two */
    }
    return s;
}

int vb200_lm::gemm(const Linear &l, Acts *in, int M, float *part, Acts *swiglu_out, LmPart *out) {
    if (f32()) {
        float *y = l.swiglu ? swiglu_out->rows : part;
        const int ld = l.swiglu ? swiglu_out->Kp : l.N;
        if (out) *out = {part, 1, l.N, 0};
        return lm_gemm_f32(y, ld, in->rows, in->Kp, l.W, l.Kp, M, l.N, l.K, l.swiglu ? LM_ACT_SWIGLU : LM_ACT_NONE, st);
    }
    TcActs *a = map_of(in, M);
    if (!a) return -1;
    TcGemm g;
    g.M = M;
    g.status = status;
    if (l.swiglu) {
        g.epi = TC_EPI_SWIGLU_TERMS;
        g.out_terms = swiglu_out->terms;
        g.out_rows_pad = a->rows_pad;
    } else if (fused_act(l, M)) {
        g.epi = TC_EPI_RELU2_TERMS;
        g.out = part;
        g.ld_out = g.act_n0 = l.act_n0;
        g.out_terms = l.act_acts->terms;
        g.out_terms_ld = l.act_acts->Kp;
        g.out_col0 = l.act_col;
        g.out_rows_pad = a->rows_pad;
        *out = {part, 1, l.act_n0, 0};
    } else {
        g.epi = TC_EPI_PARTIAL;
        g.splits = splits_of(l, M);
        g.out = part;
        g.ld_out = l.N;
        *out = {part, g.splits, l.N, (size_t)M * l.N};
    }
    return tc_gemm(l.tc, *a, g, st);
}

/* The in-projection is done up to here; a stretch's keys and values are written out and attended to. */
int vb200_lm::latent_wide(const Layer &l, const LmMixer &m, const LmLatent &a, const RunState &s, int M) {
    const int first = m.mask.window > 0 ? std::max(0, pos_now - m.mask.window + 1) : 0, n = pos_now + M - first;
    const int rp = n <= 256 ? 256 : round_up(n, 128);
    Acts *c = l.mix.kv_acts;
    if (gathered.acts != c || gathered.cache != s.a || gathered.first != first || gathered.n != n) {
        LM_DO(lm_latent_gather(a, c->terms, rp, c->Kp, first, n, st));
        gathered.acts = c;
        gathered.cache = s.a;
        gathered.first = first;
        gathered.n = n;
    }
    TcActs map;
    if (tc_acts_blocks(&map, c->terms, rp, c->Kp)) return fail("tensor map of the latents could not be made");
    TcGemm g;
    g.M = n;
    g.epi = TC_EPI_TERMS;
    g.status = status;
    g.out_terms = wide;
    g.out_rows_pad = rp;
    g.out_terms_ld = l.mix.ukv.N;
    LM_DO(tc_gemm(l.mix.ukv.tc, map, g, st));
    LmAttn t = {};
    t.dyn = dyn();
    t.heads = t.kv_heads = m.heads; t.dim = m.dim + m.rot_dim; t.vdim = m.vdim;
    t.window = m.mask.window; t.scale = (float)m.scale; t.rot = m.rope.dims;
    t.ring = s.ring;
    t.out = a.out;
    LmWide w = {};
    w.kv = wide; w.plane = (size_t)rp * l.mix.ukv.N; w.ld = l.mix.ukv.N; w.v0 = m.heads * m.dim; w.first = first;
    w.cache = slabs + s.a; w.slab = slab; w.rank = m.kv_rank; w.rot_dim = m.rot_dim;
    w.q = a.q; w.cs = cs; w.gate = gate;
    LM_DO(lm_attn_wide(t, w, M, st));
    return 0;
}

/* x_acts hold the normed rows; leaves the rows of the out-projection. */
int vb200_lm::latent(const Layer &l, const LmLayer &spec, const RunState &s, int M) {
    const LmMixer &m = spec.mixer;
    LmLatent a = {};
    LM_DO(gemm(l.mix.in, x_acts, M, part_in, nullptr, &a.in));
    a.dyn = dyn();
    a.heads = m.heads; a.dim = m.dim; a.rot_dim = m.rot_dim; a.vdim = m.vdim; a.rank = m.kv_rank; a.q_rank = m.q_rank;
    a.window = m.mask.window; a.scale = (float)m.scale;
    a.rot = m.rope.dims; a.freq = l.mix.freq; a.mag = l.mix.mag; a.eps = (float)cfg.eps;
    a.q_gain = l.mix.q_gain; a.c_gain = l.mix.c_gain;
    a.ring = s.ring;
    a.kv = {slabs + s.a, slab};
    a.split = latent_split(m);
    a.col_c = l.mix.col_c; a.col_g = l.mix.col_g;
    a.q_latent = sink(l.mix.uq_acts, M);
    a.gate = gate; a.cs = cs;
    if (cfg.block == LM_BLOCK_PARALLEL && spec.mlp.experts > 0) {
        a.col_router = l.mix.col_router; a.experts = spec.mlp.experts; a.top = spec.mlp.top;
        a.chosen = route; a.weight = route_weight;
    }
    if (l.mix.in.act_n0 > 0 && !fused_act(l.mix.in, M)) { a.col_ff = l.mix.in.act_n0; a.ff = spec.mlp.ff; a.ff_out = l.mix.in.act_col; }
    a.out = sink(l.mix.acts, M);
    a.ukv = {l.mix.ukv.W, l.mix.ukv.Kp, f32() ? 0 : 1};
    a.ql = ql; a.scratch = scratch;
    LM_DO(lm_latent_prepare(a, M, st));
    LM_DO(gemm(l.mix.uq, l.mix.uq_acts, M, part_q, nullptr, &a.q));
    if (M > kLmLatentRows && latent_wide_ok(m)) return latent_wide(l, m, a, s, M);
    LM_DO(lm_latent_absorb(a, M, st));
    LM_DO(lm_latent_attend(a, M, st));
    LM_DO(lm_latent_readout(a, M, st));
    return 0;
}

/* The experts' results of the rows in x_acts, for the residual kernel to add up. */
int vb200_lm::experts(const Layer &l, const LmMlp &m, int M, LmMix *mix) {
    LmMoe e = {};
    e.experts = m.experts; e.top = m.top; e.ff = m.ff; e.width = cfg.width;
    e.chosen = route;
    e.up = {l.up.W, l.up.Kp, f32() ? 0 : 1};
    e.down = {l.down.W, l.down.Kp, f32() ? 0 : 1};
    e.x = sink(x_acts, M);
    e.act = few_act; e.act_ld = round_up(m.ff, kTcBlockK);
    e.table = route_table; e.at = route_at;
    e.y = expert_y; e.y_ld = y_ld;
    *mix = {expert_y, y_ld, m.top, route_at, route_weight};
    if (M <= kLmMoeRows) {
        LM_DO(lm_moe_few(e, M, st));
        return 0;
    }
    const int blocks = lm_moe_blocks(M, m.experts, m.top);
    Acts *ff = expert_acts[m.ff];
    LmSink to = {};
    to.rows = sorted_acts->rows; to.terms = sorted_acts->terms;
    to.rows_pad = round_up(std::max(sorted_rows, 256), 128); to.ld = sorted_acts->Kp; to.n_terms = 2;
    LM_DO(lm_moe_plan(e, M, st));
    LM_DO(lm_moe_gather(e, to, M, st));
    if (f32()) {
        LM_DO(lm_gemm_f32(ff->rows, ff->Kp, to.rows, to.ld, l.up.W, l.up.Kp, blocks * 128, m.ff, cfg.width, LM_ACT_RELU2, st, route_table,
                          l.expert_rows));
        LM_DO(lm_gemm_f32(expert_y, y_ld, ff->rows, ff->Kp, l.down.W, l.down.Kp, blocks * 128, cfg.width, m.ff, LM_ACT_NONE, st, route_table,
                          l.expert_rows_down));
        return 0;
    }
    TcActs xa, fa;
    if (tc_acts_blocks(&xa, to.terms, to.rows_pad, to.ld) || tc_acts_blocks(&fa, ff->terms, to.rows_pad, ff->Kp))
        return fail("tensor map of the experts' rows could not be made");
    TcGemm g;
    g.status = status;
    g.epi = TC_EPI_RELU2_TERMS;
    g.out_terms = ff->terms; g.out_terms_ld = ff->Kp; g.out_rows_pad = to.rows_pad;
    LM_DO(tc_gemm_grouped(l.up.tc, xa, g, m.ff, route_table, blocks, st));
    g = TcGemm();
    g.status = status;
    g.epi = TC_EPI_STORE;
    g.out = expert_y; g.ld_out = y_ld;
    LM_DO(tc_gemm_grouped(l.down.tc, fa, g, cfg.width, route_table, blocks, st));
    return 0;
}

/* x_acts hold the normed rows; leaves the rows of the out-projection. */
int vb200_lm::mixer(const Layer &l, const LmLayer &spec, const RunState &s, int M) {
    const LmMixer &m = spec.mixer;
    if (m.kind == LM_MIXER_LATENT) return latent(l, spec, s, M);
    LmPart in;
    LM_DO(gemm(l.mix.in, x_acts, M, part_in, nullptr, &in));
    if (m.kind == LM_MIXER_ATTENTION) {
        LmAttn a = {};
        a.dyn = dyn();
        a.heads = m.heads; a.kv_heads = m.kv_heads; a.dim = m.dim; a.vdim = m.vdim;
        a.window = m.mask.window; a.keep = m.mask.keep_first;
        a.scale = (float)m.scale; a.softcap = (float)m.softcap;
        a.rot = m.rope.dims; a.freq = l.mix.freq; a.mag = l.mix.mag;
        a.q_gain = l.mix.q_gain; a.k_gain = l.mix.k_gain; a.eps = (float)cfg.eps;
        a.ring = s.ring;
        a.k = {slabs + s.a, slab}; a.v = {slabs + s.b, slab};
        a.split = !f32() && lm_attn_mma_ok(m.dim, m.vdim);
        a.qkv = in; a.q = q; a.scratch = scratch; a.tickets = tickets;
        a.out = sink(l.mix.acts, M);
        if (M == 1 && lm_attn_step_ok(a)) {
            LM_DO(lm_attn_step(a, st));
        } else {
            LM_DO(lm_attn_prepare(a, M, st));
            if (a.split && M > 8) LM_DO(lm_attn_mma(a, M, st));
            else LM_DO(lm_attn_generic(a, M, st));
        }
    } else {
        LmDelta d = {};
        d.dyn = dyn();
        d.heads = m.heads; d.kv_heads = m.kv_heads; d.dim = m.dim; d.vdim = m.vdim; d.taps = m.taps;
        d.eps = (float)cfg.eps;
        d.conv = l.mix.conv; d.decay = l.mix.decay; d.dt_bias = l.mix.dt_bias; d.norm = l.mix.norm;
        d.s = {slabs + s.a, slab}; d.tail = {slabs + s.b, slab};
        d.in = in; d.q = q; d.k = k; d.v = v; d.beta = beta; d.decays = decays; d.gram = gram; d.o = o; d.status = status;
        d.out = sink(l.mix.acts, M);
        if (M == 1 && lm_delta_step_ok(d)) {
            LM_DO(lm_delta_step(d, st));
        } else {
            LM_DO(lm_delta_inputs(d, M, st));
            LM_DO(lm_delta_scan(d, M, st));
            LM_DO(lm_delta_gate(d, M, st));
        }
    }
    return 0;
}

/* All launches of M rows (d_in holds position, tokens and wanted rows). logits_out: host rows. */
int vb200_lm::enqueue(int M, int n_want, float *logits_out, bool greedy) {
    LmPart out = {};
    LmResidual r = {};
    r.dyn = dyn(); r.tokens = tokens(); r.embed = embed; r.width = cfg.width; r.eps = (float)cfg.eps; r.x = x;
    r.rms = cfg.norm == LM_NORM_RMS;
    gathered = {};
    auto next = [&](size_t i) {          /* what the residual kernel before run i prepares */
        if (runs[i].begins_pass) { r.next = LM_NEXT_CONCAT; r.sink = sink(loop_acts, M); }
        else { r.next = LM_NEXT_NORM; r.next_gain = layers[runs[i].layer].norm1; r.sink = sink(x_acts, M); }
    };
    r.first = 1;
    next(0);
    LM_DO(lm_residual(r, M, st));
    r.first = 0;
    for (size_t i = 0; i < runs.size(); i++) {
        const Layer &l = layers[runs[i].layer];
        if (runs[i].begins_pass) {
            LM_DO(gemm(loop_in, loop_acts, M, part_out, nullptr, &out));
            r.part = out; r.join = LM_JOIN_REPLACE;
            r.next = LM_NEXT_NORM; r.next_gain = l.norm1; r.sink = sink(x_acts, M);
            LM_DO(lm_residual(r, M, st));
        }
        const LmLayer &spec = cfg.layers[runs[i].layer];
        if (mixer(l, spec, states[i], M)) return -1;
        r.mix.top = 0;
        if (cfg.block == LM_BLOCK_PARALLEL && spec.mlp.experts > 0 && experts(l, spec.mlp, M, &r.mix)) return -1;
        LM_DO(gemm(l.mix.out, l.mix.acts, M, part_out, nullptr, &out));
        r.part = out; r.join = cfg.block == LM_BLOCK_PARALLEL ? LM_JOIN_ADD : LM_JOIN_NORMED; r.post_gain = l.norm1b;
        if (l.ff_acts) {
            r.next = LM_NEXT_NORM; r.next_gain = l.norm2; r.sink = sink(x_acts, M);
            LM_DO(lm_residual(r, M, st));
            LM_DO(gemm(l.up, x_acts, M, nullptr, l.ff_acts, nullptr));
            LM_DO(gemm(l.down, l.ff_acts, M, part_out, nullptr, &out));
            r.part = out; r.post_gain = l.norm2b;
        }
        if (i + 1 < runs.size()) {
            next(i + 1);
            r.tap = tap_on ? tap + i * (size_t)block * cfg.width : nullptr;
            LM_DO(lm_residual(r, M, st));
            r.tap = nullptr;
        }
    }
    /* the head sees the wanted rows only */
    LmPart lg = {};
    for (int w0 = 0; w0 < n_want; w0 += kHeadRows) {
        const int nw = std::min(n_want - w0, kHeadRows);
        r.row_of = greedy && M == 1 ? zero : wanted() + w0;
        r.next = LM_NEXT_NORM; r.next_gain = final_norm; r.sink = sink(x_acts, nw);
        LM_DO(lm_residual(r, nw, st));
        LM_DO(gemm(head, x_acts, nw, part_head, nullptr, &lg));
        if (greedy) {
            LM_DO(lm_argmax_advance(dyn(), tokens(), log, kLogCap, lg, cfg.vocab, M, st));
        } else {
            tc_reduce(logits, lg.p, lg.n, lg.stride, (size_t)nw * lg.ld, nullptr, lg.ld, st);
            if (logits_out)
                LM_CUDA(cudaMemcpy2DAsync(logits_out + (size_t)w0 * cfg.vocab, sizeof(float) * cfg.vocab, logits, sizeof(float) * lg.ld,
                                          sizeof(float) * cfg.vocab, nw, cudaMemcpyDeviceToHost, st));
        }
    }
    if (tap_on) {
        r.row_of = nullptr;
        r.next = LM_NEXT_NONE;
        r.tap = tap + (runs.size() - 1) * (size_t)block * cfg.width;
        LM_DO(lm_residual(r, M, st));
        tap_rows = M;
    }
    return 0;
}

/* One-token steps: the first call of a variant runs launch by launch (kernel attributes are set on
 * first use, which must not happen inside a capture), the second is captured, later ones replay. */
int vb200_lm::launch(int M, int n_want, float *logits_out, bool greedy) {
    if (M != 1 || tap_on || f32()) return enqueue(M, n_want, logits_out, greedy);
    const int v = greedy ? STEP_GREEDY : n_want ? STEP_LOGITS : STEP_SILENT;
    if (!exec[v]) {
        if (direct_calls[v]++ == 0) return enqueue(M, n_want, logits_out, greedy);
        cudaGraph_t graph = nullptr;
        LM_CUDA(cudaStreamBeginCapture(st, cudaStreamCaptureModeRelaxed));
        const int rc = enqueue(M, n_want, nullptr, greedy);
        const cudaError_t ee = cudaStreamEndCapture(st, &graph);
        if (rc || ee != cudaSuccess || !graph) {
            if (graph) cudaGraphDestroy(graph);
            cudaGetLastError();
            return rc ? -1 : fail("the one-token step could not be captured");
        }
        const cudaError_t ie = cudaGraphInstantiate(&exec[v], graph, 0);
        cudaGraphDestroy(graph);
        if (ie != cudaSuccess) {
            exec[v] = nullptr;
            return cuda_ok(ie, "cudaGraphInstantiate");
        }
    }
    LM_CUDA(cudaGraphLaunch(exec[v], st));
    if (v == STEP_LOGITS && logits_out)
        LM_CUDA(cudaMemcpyAsync(logits_out, logits, sizeof(float) * cfg.vocab, cudaMemcpyDeviceToHost, st));
    return 0;
}

/* Position, tokens and wanted rows of the next M rows to the device. */
int vb200_lm::feed(int seq, const int *tok, int M, const int *want, int n_want) {
    const int b = in_next;
    in_next ^= 1;
    if (in_busy[b]) LM_CUDA(cudaEventSynchronize(in_free[b]));
    int *h = h_in[b];
    LmDyn d = {seq, seqs[seq].length, 0, 0};
    pos_now = seqs[seq].length;
    memcpy(h, &d, sizeof(d));
    memcpy(h + 4, tok, sizeof(int) * M);
    if (n_want) memcpy(h + 4 + block, want, sizeof(int) * n_want);
    LM_CUDA(cudaMemcpyAsync(d_in, h, sizeof(int) * (n_want ? 4 + block + n_want : 4 + M), cudaMemcpyHostToDevice, st));
    LM_CUDA(cudaEventRecord(in_free[b], st));
    in_busy[b] = true;
    return 0;
}

int vb200_lm::finish() {
    int s = 0;
    LM_CUDA(cudaMemcpyAsync(&s, status, sizeof(int), cudaMemcpyDeviceToHost, st));
    LM_CUDA(cudaStreamSynchronize(st));
    if (s) {
        cudaMemsetAsync(status, 0, sizeof(int), st);
        return fail("a bounded wait ran out on the device (status " + std::to_string(s) + ")");
    }
    return 0;
}

/* ------------------------------------------------------------------ C ABI */
static vb200_lm_t *open_with(LmConfig &&cfg, const Source &src, const vb200_lm_options_t *opt) {
    std::unique_ptr<vb200_lm> lm(new vb200_lm());
    lm->cfg = std::move(cfg);
    return lm->init(src, opt) ? nullptr : lm.release();
}

static bool read_text(const std::string &path, std::string *out) {
    FILE *f = fopen(path.c_str(), "rb");
    if (!f) return false;
    char buf[65536];
    size_t n;
    while ((n = fread(buf, 1, sizeof(buf), f)) > 0) out->append(buf, n);
    fclose(f);
    return true;
}

static int check_step(vb200_lm *lm, int seq, const int *tokens, int n) {
    if (!lm) return fail("no model");
    if (seq < 0 || seq >= lm->max_seqs || !lm->seqs[seq].open) return fail("no such open sequence");
    if (n < 1 || !tokens) return fail("a step needs at least one token");
    if (lm->seqs[seq].length + (long long)n > lm->max_tokens) return fail("the sequence would exceed max_tokens");
    for (int i = 0; i < n; i++)
        if (tokens[i] < 0 || tokens[i] >= lm->cfg.vocab) return fail("token " + std::to_string(tokens[i]) + " is outside the vocabulary");
    return 0;
}

extern "C" {

const char *vb200_lm_error(void) { return g_error.c_str(); }

int vb200_lm_check_config(const char *config_json) {
    LmConfig c;
    std::string err;
    g_error.clear();
    if (!config_json || !lm_config_from_text(config_json, &c, &err)) return fail(err);
    return check_sizes(c);
}

vb200_lm_t *vb200_lm_open(const char *model_dir, const vb200_lm_options_t *opt) {
    g_error.clear();
    LmConfig cfg;
    std::string text, err;
    const std::string dir = model_dir ? model_dir : "";
    if (!read_text(dir + "/config.json", &text)) { fail(dir + "/config.json cannot be read"); return nullptr; }
    if (!lm_config_from_text(text, &cfg, &err)) { fail(err); return nullptr; }
    SafeTensors file;
    if (!file.open((dir + "/model.safetensors").c_str(), &err)) { fail(err); return nullptr; }
    Source s;
    s.file = &file;
    return open_with(std::move(cfg), s, opt);
}

vb200_lm_t *vb200_lm_open_random(const char *config_json, const vb200_lm_options_t *opt, unsigned seed) {
    g_error.clear();
    LmConfig cfg;
    std::string err;
    if (!config_json || !lm_config_from_text(config_json, &cfg, &err)) { fail(err); return nullptr; }
    Source s;
    s.seed = seed;
    return open_with(std::move(cfg), s, opt);
}

void vb200_lm_close(vb200_lm_t *lm) { delete lm; }

int vb200_lm_info(vb200_lm_t *lm, vb200_lm_info_t *i) {
    if (!lm || !i) return -1;
    i->vocab = lm->cfg.vocab; i->width = lm->cfg.width;
    i->layers = (int)lm->cfg.layers.size(); i->runs = (int)lm->runs.size();
    i->max_seqs = lm->max_seqs; i->max_tokens = lm->max_tokens; i->block_rows = lm->block; i->dtype = lm->dtype;
    i->weight_bytes = lm->weight_bytes;
    i->state_bytes_per_seq = lm->slab * sizeof(float);
    return 0;
}

int vb200_lm_seq_open(vb200_lm_t *lm) {
    if (!lm) return fail("no model");
    for (int i = 0; i < lm->max_seqs; i++)
        if (!lm->seqs[i].open) {
            lm->seqs[i] = {true, 0};
            return i;
        }
    return fail("every slot is taken");
}

int vb200_lm_seq_close(vb200_lm_t *lm, int seq) {
    if (!lm || seq < 0 || seq >= lm->max_seqs || !lm->seqs[seq].open) return fail("no such open sequence");
    lm->seqs[seq] = {false, 0};
    return 0;
}

int vb200_lm_seq_length(vb200_lm_t *lm, int seq) {
    if (!lm || seq < 0 || seq >= lm->max_seqs || !lm->seqs[seq].open) return fail("no such open sequence");
    return lm->seqs[seq].length;
}

int vb200_lm_step(vb200_lm_t *lm, int seq, const int *tokens, int n, const int *want, int n_want, float *logits_out) {
    g_error.clear();
    if (check_step(lm, seq, tokens, n)) return -1;
    if (n_want < 0 || (n_want && (!want || !logits_out))) return fail("wanted places without a buffer");
    for (int i = 0; i < n_want; i++)
        if (want[i] < 0 || want[i] >= n || (i && want[i] <= want[i - 1])) return fail("wanted places have to ascend inside the portion");
    if (lm->tap_on && n > lm->block) return fail("a tapped step has at most block_rows tokens");
    int w = 0;
    std::vector<int> local;
    for (int r0 = 0; r0 < n; r0 += lm->block) {
        const int M = std::min(lm->block, n - r0), w0 = w;
        local.clear();
        for (; w < n_want && want[w] < r0 + M; w++) local.push_back(want[w] - r0);
        if (lm->feed(seq, tokens + r0, M, local.data(), (int)local.size())) return -1;
        if (lm->launch(M, (int)local.size(), logits_out + (size_t)w0 * lm->cfg.vocab, false)) return -1;
        lm->seqs[seq].length += M;
    }
    return lm->finish();
}

int vb200_lm_generate(vb200_lm_t *lm, int seq, const int *prompt, int n, int n_new, int *out) {
    g_error.clear();
    if (check_step(lm, seq, prompt, n)) return -1;
    if (n_new < 1 || n_new > kLogCap || !out) return fail("number of new tokens out of range");
    if (lm->tap_on) return fail("generation runs without the residual-stream tap");
    if (lm->seqs[seq].length + (long long)n + n_new - 1 > lm->max_tokens) return fail("the sequence would exceed max_tokens");
    cudaEventRecord(lm->ev[0], lm->st);
    for (int r0 = 0; r0 < n; r0 += lm->block) {
        const int M = std::min(lm->block, n - r0), last = M - 1;
        const bool end = r0 + M == n;
        if (lm->feed(seq, prompt + r0, M, &last, end ? 1 : 0)) return -1;
        if (lm->launch(M, end ? 1 : 0, nullptr, end)) return -1;
        lm->seqs[seq].length += M;
    }
    cudaEventRecord(lm->ev[1], lm->st);
    /* position, token and log are on the device from here on */
    for (int i = 1; i < n_new; i++) {
        if (lm->launch(1, 1, nullptr, true)) return -1;
        lm->seqs[seq].length += 1;
    }
    cudaEventRecord(lm->ev[2], lm->st);
    LM_CUDA(cudaMemcpyAsync(out, lm->log, sizeof(int) * n_new, cudaMemcpyDeviceToHost, lm->st));
    lm->timed = true;
    return lm->finish() ? -1 : n_new;
}

int vb200_lm_last_ms(vb200_lm_t *lm, float *prompt_ms, float *decode_ms) {
    if (!lm || !lm->timed) return fail("nothing was generated yet");
    if (prompt_ms) LM_CUDA(cudaEventElapsedTime(prompt_ms, lm->ev[0], lm->ev[1]));
    if (decode_ms) LM_CUDA(cudaEventElapsedTime(decode_ms, lm->ev[1], lm->ev[2]));
    return 0;
}

int vb200_lm_tap_enable(vb200_lm_t *lm, int on) {
    if (!lm) return fail("no model");
    if (on && !lm->tap) {
        void *p = nullptr;
        if (cudaMalloc(&p, sizeof(float) * lm->runs.size() * (size_t)lm->block * lm->cfg.width) != cudaSuccess) {
            cudaGetLastError();
            return fail("out of device memory for the tap");
        }
        lm->allocs.push_back(p);
        lm->tap = (float *)p;
    }
    lm->tap_on = on != 0;
    return 0;
}

int vb200_lm_tap_read(vb200_lm_t *lm, float *out, int n) {
    if (!lm || !lm->tap || !out || n < 1 || n > lm->tap_rows) return fail("no tapped step of that length");
    const size_t W = sizeof(float) * lm->cfg.width;
    LM_CUDA(cudaStreamSynchronize(lm->st));
    LM_CUDA(cudaMemcpy2D(out, W * n, lm->tap, W * lm->block, W * n, lm->runs.size(), cudaMemcpyDeviceToHost));
    return 0;
}

} // extern "C"
