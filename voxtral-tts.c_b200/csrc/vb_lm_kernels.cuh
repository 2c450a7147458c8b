/*
 * vb_lm_kernels.cuh - device side of the decoder language models: argument blocks and launchers
 * of the kernels between the GEMMs (vb_lm_kernels.cu, vb_lm_attn.cu, vb_lm_latent.cu, vb_lm_delta.cu,
 * vb_lm_moe.cu).
 *
 * A kernel reads the result of a GEMM as split-K partials (LmPart), and leaves rows for the next
 * one in an LmSink: BF16 terms for the tensor-core GEMM, or plain fp32 rows for the fp32 one.
 * Everything in between is fp32. Where a sequence stands, and in which slot, is read from device
 * memory (LmDyn), so that a captured graph serves every position and slot.
 */
#ifndef VB_LM_KERNELS_CUH
#define VB_LM_KERNELS_CUH

#include <cuda_runtime.h>
#include <stdint.h>

#include "vb_common.cuh"

namespace vb {

struct LmDyn {
    int slot;      /* whose cache and state */
    int pos;       /* position of the first row of this launch sequence */
    int logged;    /* tokens written by the generation loop */
    int pad;
};

constexpr int kLmMaxParts = 8;   /* split-K factor limit of the GEMM */

/* Split-K partials of a GEMM: n buffers [M][ld], stride floats apart; their sum is the result. */
struct LmPart {
    const float *p;
    int n, ld;
    size_t stride;
};

VB_DEVINL float lm_sum(const LmPart &g, int m, int c) {
    const float *q = g.p + (size_t)m * g.ld + c;
    float v = __ldcg(q);
    for (int i = 1; i < g.n; i++) v += __ldcg(q + (size_t)i * g.stride);
    return v;
}

/* The same with every partial requested before the first is used. */
VB_DEVINL float lm_sum_batch(const LmPart &g, int m, int c) {
    const float *q = g.p + (size_t)m * g.ld + c;
    float t[kLmMaxParts], v = 0.0f;
#pragma unroll
    for (int i = 0; i < kLmMaxParts; i++) t[i] = i < g.n ? __ldcg(q + (size_t)i * g.stride) : 0.0f;
#pragma unroll
    for (int i = 0; i < kLmMaxParts; i++) v += t[i];
    return v;
}
/* Two columns from c on (c and ld even). */
VB_DEVINL float2 lm_sum2(const LmPart &g, int m, int c) {
    const float *q = g.p + (size_t)m * g.ld + c;
    float2 v = __ldcg(reinterpret_cast<const float2 *>(q));
    for (int i = 1; i < g.n; i++) {
        const float2 t = __ldcg(reinterpret_cast<const float2 *>(q + (size_t)i * g.stride));
        v.x += t.x;
        v.y += t.y;
    }
    return v;
}
/* Four columns from c on (c and ld multiples of 4). */
VB_DEVINL float4 lm_sum4(const LmPart &g, int m, int c) {
    const float *q = g.p + (size_t)m * g.ld + c;
    float4 t[kLmMaxParts];
#pragma unroll
    for (int i = 0; i < kLmMaxParts; i++)
        t[i] = i < g.n ? __ldcg(reinterpret_cast<const float4 *>(q + (size_t)i * g.stride)) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int i = 1; i < kLmMaxParts; i++)
        if (i < g.n) { t[0].x += t[i].x; t[0].y += t[i].y; t[0].z += t[i].z; t[0].w += t[i].w; }
    return t[0];
}

/* Activation rows of the next GEMM. */
struct LmSink {
    float *rows;        /* fp32 rows [M][ld], or null */
    uint16_t *terms;    /* BF16 terms [n_terms][rows_pad][ld], or null */
    int rows_pad, ld, n_terms;
};

VB_DEVINL void lm_put(const LmSink &s, int m, int c, float v) {
    if (s.rows) {
        s.rows[(size_t)m * s.ld + c] = v;
    } else {
        uint16_t t0, t1, t2;
        vb_split3(v, t0, t1, t2);
        uint16_t *o = s.terms + (size_t)m * s.ld + c;
        const size_t term = (size_t)s.rows_pad * s.ld;
        o[0] = t0;
        if (s.n_terms > 1) o[term] = t1;
        if (s.n_terms > 2) o[2 * term] = t2;
    }
}

/* Four columns from c on (a multiple of 4; rows are padded to multiples of 64). */
VB_DEVINL void lm_put4(const LmSink &s, int m, int c, const float (&v)[4]) {
    if (s.rows) {
        *reinterpret_cast<float4 *>(s.rows + (size_t)m * s.ld + c) = make_float4(v[0], v[1], v[2], v[3]);
    } else {
        uint16_t t[3][4];
#pragma unroll
        for (int i = 0; i < 4; i++) vb_split3(v[i], t[0][i], t[1][i], t[2][i]);
        uint16_t *o = s.terms + (size_t)m * s.ld + c;
        const size_t term = (size_t)s.rows_pad * s.ld;
#pragma unroll
        for (int j = 0; j < 3; j++)
            if (j < s.n_terms)
                *reinterpret_cast<uint2 *>(o + j * term) = make_uint2(t[j][0] | ((uint32_t)t[j][1] << 16), t[j][2] | ((uint32_t)t[j][3] << 16));
    }
}

/* State of one layer run: `base` + slot * `slab` floats. */
struct LmState {
    float *base;
    size_t slab;
};
VB_DEVINL float *lm_state(const LmState &s, const LmDyn *dyn) { return s.base + (size_t)dyn->slot * s.slab; }

/* Where position p of a windowed layer lives: the first `keep` positions have rows of their own,
 * the others share a ring. (An unwindowed layer is a ring that never wraps.) */
struct LmRing {
    int keep, ring;
};
VB_DEVINL int lm_ring_row(const LmRing &r, int p) { return p < r.keep ? p : r.keep + (p - r.keep) % r.ring; }

/* Elements of a weight matrix as it is kept: in tiles of 128 rows x 64 columns for the tensor cores, or row by
 * row. lm_weight_row: 64 columns (block kb of a row of Kp) that lie together. */
struct LmWeight {
    const uint16_t *W;
    int Kp, tiled;
};
VB_DEVINL const uint16_t *lm_weight_row(const LmWeight &w, int n, int kb) {
    return w.tiled ? w.W + (((size_t)(n >> 7) * (w.Kp >> 6) + kb) * 128 + (n & 127)) * 64 : w.W + (size_t)n * w.Kp + kb * 64;
}

/* Results of the experts of a mixture: row at[m * top + k] of y belongs to the k-th choice of token m. */
struct LmMix {
    const float *y;
    int ld, top;                 /* top 0: no mixture */
    const int *at;
    const float *weight;         /* [M][top] */
};

/* ---- residual stream (vb_lm_kernels.cu) ---- */
enum LmNext { LM_NEXT_NONE = 0, LM_NEXT_NORM = 1, LM_NEXT_CONCAT = 2 };
enum LmJoin { LM_JOIN_REPLACE = 0, LM_JOIN_NORMED = 1, LM_JOIN_ADD = 2 };

struct LmResidual {
    const LmDyn *dyn;
    const int *tokens;           /* [M] */
    const uint16_t *embed;       /* [vocab][width] BF16 */
    int width;
    float eps;
    int first;                   /* 1: x = embedding of the row's token (part unused) */
    int rms;                     /* norms divide by the root mean square; 0: they centre first */
    LmPart part;                 /* sublayer output */
    int join;                    /* LmJoin: x = part, x += norm(part) * post_gain, x += part (+ mix) */
    const float *post_gain;
    LmMix mix;
    float *x;                    /* [M][width] residual stream, in and out */
    const int *row_of;           /* optional: output row m takes row row_of[m] of part and x (x is then not stored) */
    float *tap;                  /* optional copy of the new x, [M][width] */
    int next;                    /* LmNext: what goes to the sink */
    const float *next_gain;      /* LM_NEXT_NORM */
    LmSink sink;
};
int lm_residual(const LmResidual &a, int M, cudaStream_t st);

/* Weight repacking: row r of src [rows][K] goes to row row0 + r * step of dst [..][Kp], from column col0 on. */
int lm_pack_rows(uint16_t *dst, int Kp, int row0, int step, int col0, const uint16_t *src, int rows, int K, cudaStream_t st);
int lm_widen(float *dst, const uint16_t *src, int n, cudaStream_t st);
int lm_fill_random(uint16_t *dst, size_t n, uint32_t seed, float mean, float scale, cudaStream_t st);

/* fp32 GEMM on the fp32 pipes: y[M][ld_out] = x[M][ldx] . W[N][ldw]^T, BF16 W. LM_ACT_SWIGLU: rows of W
 * interleaved (gate, up), y[M][N / 2] = silu(gate) * up. With a table of row blocks (as for tc_gemm_grouped, M = 128 times
 * their number) a block uses the matrix that starts at row matrix * group_rows of W. */
enum LmAct { LM_ACT_NONE = 0, LM_ACT_SWIGLU = 1, LM_ACT_RELU2 = 2 };
int lm_gemm_f32(float *y, int ld_out, const float *x, int ldx, const uint16_t *W, int ldw, int M, int N, int K, LmAct act,
                cudaStream_t st, const int4 *table = nullptr, int group_rows = 0);

/* Largest logit of row 0 (first one on a tie) becomes the next token: tokens[0], log[dyn->logged++];
 * the sequence moves on by the `rows` positions just run. */
int lm_argmax_advance(LmDyn *dyn, int *tokens, int *log, int log_cap, LmPart logits, int vocab, int rows, cudaStream_t st);

/* ---- attention (vb_lm_attn.cu) ---- */
struct LmAttn {
    const LmDyn *dyn;
    int heads, kv_heads, dim, vdim;
    int window, keep;            /* window 0: every earlier key */
    float scale, softcap;        /* softcap 0: none */
    int rot;                     /* rotated dimensions */
    const float *freq;           /* [2][rot / 2]: angle per position, high and low part */
    float mag;
    const float *q_gain, *k_gain;
    float eps;
    LmRing ring;
    LmState k, v;                /* [ring rows][kv_heads * dim], [..][kv_heads * vdim] */
    int split;                   /* 1: a head's part of a cache row is [size] BF16 high halves, then [size] low halves
                                    (hi + lo carry 16 mantissa bits), ready for the tensor cores; 0: fp32 */
    LmPart qkv;
    float *q;                    /* [M][heads * dim] normed and rotated */
    float *scratch;              /* key-split partials */
    unsigned *tickets;
    LmSink out;
};
constexpr int kLmAttnSplits = 32;        /* key splits of one row's attention, at most */
constexpr int kLmAttnPairs = 16;         /* (row, head) pairs per CTA of the generic kernel */
size_t lm_attn_scratch_floats(int heads, int kv_heads, int vdim);
int lm_attn_ticket_count(int heads, int kv_heads);
int lm_attn_prepare(const LmAttn &a, int M, cudaStream_t st);              /* norm, rotation, cache append */
int lm_attn_generic(const LmAttn &a, int M, cudaStream_t st);              /* fp32 pipes, any size */
bool lm_attn_step_ok(const LmAttn &a);
int lm_attn_step(const LmAttn &a, cudaStream_t st);                        /* one token: norm, rotation, append, attention */
bool lm_attn_mma_ok(int dim, int vdim);                                    /* sizes it runs at; needs split caches */
int lm_attn_mma(const LmAttn &a, int M, cudaStream_t st);                  /* warp-level tensor cores, prompts */

/* Keys and values of every head, written out of a latent for a prompt's attention. */
struct LmWide {
    const uint16_t *kv;          /* two BF16 planes (high, low) of rows [heads * plain | heads * vdim] */
    size_t plane;                /* elements between the planes */
    int ld, v0;                  /* row length, first value column */
    int first;                   /* position of row 0 */
    const float *cache;          /* latent cache (split): rows [rank + rot_dim]; slot 0 */
    size_t slab;
    int rank, rot_dim;
    LmPart q;                    /* [M][heads * (plain + rot_dim)], not rotated */
    const float *cs;             /* [M][rot]: cosines, then sines */
    const float *gate;           /* [M][heads] */
};
bool lm_attn_wide_ok(int plain, int rot_dim, int vdim);
int lm_attn_wide(const LmAttn &a, const LmWide &w, int M, cudaStream_t st);   /* a.dim = plain + rot_dim */

/* ---- latent attention (vb_lm_latent.cu) ---- */
/* A token leaves a latent of `rank` and a rotated key part of `rot_dim` in the cache. Few rows: the query is
 * carried into the latent's space (absorb), attends over cache rows (attend, one key of rank + rot_dim per
 * token for all heads), and what it read goes through the value matrix (readout). Prompts: gather +
 * GEMM + lm_attn_wide. */
struct LmLatent {
    const LmDyn *dyn;
    int heads, dim, rot_dim, vdim, rank, q_rank;
    int window;                  /* 0: every earlier key */
    float scale;
    int rot;                     /* rotated dimensions of rot_dim, 2i paired with 2i + 1 */
    const float *freq;           /* [2][rot / 2] */
    float mag, eps;
    const float *q_gain, *c_gain;   /* c_gain null: the cache is another layer's */
    LmRing ring;
    LmState kv;                  /* [ring rows][rank + rot_dim] */
    int split;                   /* cache rows as BF16 high halves, then low halves */
    /* in-projection: query latent from column 0, the others where they begin */
    LmPart in;
    int col_c, col_g;
    LmSink q_latent;             /* normed query latent */
    float *gate, *cs;            /* [M][heads], [M][rot] */
    int col_router, experts, top;   /* experts 0: no router */
    int *chosen;                 /* [M][top], by falling logit */
    float *weight;
    int col_ff, ff, ff_out;      /* columns that go to `out` from column ff_out on as max(., 0)^2; ff 0: none */
    LmSink out;                  /* rows of the out-projection: [heads * vdim, ...] */
    LmPart q;                    /* [M][heads * (dim + rot_dim)] */
    LmWeight ukv;                /* rows [heads * dim] key part, [heads * vdim] value part */
    float *ql;                   /* [M][heads][rank + rot_dim] */
    float *scratch;              /* what the key splits leave for the readout */
};
constexpr int kLmLatentRows = 16;        /* rows that take the absorbed form where the written-out one is possible */
constexpr int kLmLatentPairs = 16;       /* (row, head) pairs per CTA */
bool lm_latent_split_ok(int rank, int rot_dim);
bool lm_latent_supported(int q_rank, int rank, int rot_dim);
size_t lm_latent_scratch_floats(int rows, int heads, int rank);
int lm_latent_prepare(const LmLatent &a, int M, cudaStream_t st);     /* norms, rotation, cache append, gates, routing */
int lm_latent_absorb(const LmLatent &a, int M, cudaStream_t st);
int lm_latent_attend(const LmLatent &a, int M, cudaStream_t st);
int lm_latent_readout(const LmLatent &a, int M, cudaStream_t st);
/* Latents of positions first .. first + n - 1 as BF16 terms [2][rows_pad][ld]. */
int lm_latent_gather(const LmLatent &a, uint16_t *terms, int rows_pad, int ld, int first, int n, cudaStream_t st);

/* ---- mixture of experts (vb_lm_moe.cu) ---- */
struct LmMoe {
    int experts, top, ff, width;
    const int *chosen;           /* [M][top] */
    LmWeight up, down;           /* the experts' matrices stacked, each padded to whole 128-row tiles */
    LmSink x;                    /* the rows the experts read */
    float *act;                  /* few rows: [M * top][padded ff] */
    int act_ld;
    /* many rows: tokens sorted by expert in blocks of 128 rows */
    int4 *table;
    int *at;                     /* [M * top]: row of a choice (few rows: its own index) */
    float *y;                    /* results, [rows][y_ld] */
    int y_ld;
};
constexpr int kLmMoeRows = 4;            /* rows that go expert by expert without sorting */
constexpr int kLmMoeExperts = 1024;
int lm_moe_blocks(int rows, int experts, int top);                    /* row blocks that M rows can need */
int lm_moe_few(const LmMoe &a, int M, cudaStream_t st);               /* both products; results in row m * top + k */
int lm_moe_plan(const LmMoe &a, int M, cudaStream_t st);              /* table and at */
int lm_moe_gather(const LmMoe &a, const LmSink &to, int M, cudaStream_t st);   /* `to`: sorted rows */

/* ---- gated delta rule (vb_lm_delta.cu) ---- */
struct LmDelta {
    const LmDyn *dyn;
    int heads, kv_heads, dim, vdim, taps;
    float eps;
    const float *conv;           /* [2 * kv_heads * dim + heads * vdim][taps] */
    const float *decay;          /* [heads]: exp(A_log) */
    const float *dt_bias;        /* [heads] */
    const float *norm;           /* [vdim] */
    LmState s;                   /* [heads][dim][vdim] */
    LmState tail;                /* [taps][channels] raw convolution inputs, position p in row p % taps */
    LmPart in;                   /* columns q, k, v, gate, b, a */
    float *q, *k, *v;            /* [M][kv_heads * dim], same, [M][heads * vdim] */
    float *beta, *decays;        /* [M][heads] */
    float *gram;                 /* [groups][kv_heads][k_t.k_j, q_t.k_j][t][j]: inner products inside groups of tokens */
    int *status;                 /* set non-zero when a bounded wait runs out */
    float *o;                    /* [M][heads * vdim] */
    LmSink out;
};
constexpr int kLmDeltaGroup = 4;         /* tokens per group of the scan */
constexpr int kLmDeltaRows = 16;         /* rows are prepared in multiples of this */
int lm_delta_channels(int heads, int kv_heads, int dim, int vdim);
int lm_delta_inputs(const LmDelta &a, int M, cudaStream_t st);             /* convolution, unit norms, step sizes, decays */
int lm_delta_scan(const LmDelta &a, int M, cudaStream_t st);               /* the recurrence, fp32 pipes */
int lm_delta_gate(const LmDelta &a, int M, cudaStream_t st);               /* head norm, gate; saves the convolution's tail */
bool lm_delta_step_ok(const LmDelta &a);
int lm_delta_step(const LmDelta &a, cudaStream_t st);                      /* one token: all of the above in one launch */
bool lm_delta_supported(int dim, int vdim);

} // namespace vb

#endif
