/*
 * vb_lm_delta.cu - decoder language models: gated delta-rule mixer.
 *
 *   q, k, v = silu(short causal convolution of the projections), q and k made unit vectors
 *   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q        (per head, fp32)
 *   out = rmsnorm(o) * silu(gate)
 *
 *   lm_delta_inputs  convolution, unit norms, step sizes beta, decays: 16 rows per CTA; inner products
 *                    of the scan's groups
 *   lm_delta_scan    the recurrence in fp32, four tokens at a time; columns of S are independent, so a CTA
 *                    owns 16 of a head's value columns, S in registers, eight or more lanes per column
 *   lm_delta_gate    head norm and gate of a row; saves the raw convolution inputs of the last rows
 *   lm_delta_step    one token in one launch: a cluster of CTAs per head, 32 value columns each
 *
 * The convolution's memory is a ring of `taps` rows indexed by position, the state S a matrix per
 * head; both read as zero at the start of a sequence, so a slot needs no clearing.
 */
#include "vb_lm_kernels.cuh"
#include "vb_tc.cuh"

#include <cooperative_groups.h>

namespace vb {

namespace {

inline int ok(cudaError_t e) { return e == cudaSuccess ? 0 : -1; }

VB_DEVINL float silu(float z) { return z / (1.0f + expf(-z)); }
VB_DEVINL float softplus(float z) { return fmaxf(z, 0.0f) + log1pf(expf(-fabsf(z))); }

/* ------------------------------------------------------------------ inputs of the recurrence */
constexpr int kScGroup = kLmDeltaGroup, kGramRow = 2 * kScGroup * kScGroup;
constexpr int kInThreads = 128, kInRows = kLmDeltaRows;

/* Short convolution and silu of `size` channels from c0 on, rows [r0, r0 + rows): out[row][ld_out].
 * `raw` is room for the inputs, earlier tokens included. */
VB_DEVINL void conv_rows(const LmDelta &a, float *raw, float *out, int ld_out, int c0, int size, int r0, int rows, const float *tail,
                         int ch, int pos0) {
    const int tid = threadIdx.x, past = a.taps - 1;
    auto past_row = [&](int r, int c) {          /* an earlier token's input, zero before the sequence's start */
        return pos0 + r >= 0 ? tail[(size_t)((pos0 + r) % a.taps) * ch + c] : 0.0f;
    };
    if (((c0 | size) & 3) == 0) {
        const int per = size / 4;
        for (int i = tid; i < (past + rows) * per; i += kInThreads) {
            const int r = r0 - past + i / per, d = i % per * 4, c = c0 + d;
            *reinterpret_cast<float4 *>(raw + (i / per) * size + d) =
                r >= 0 ? lm_sum4(a.in, r, c) : make_float4(past_row(r, c), past_row(r, c + 1), past_row(r, c + 2), past_row(r, c + 3));
        }
    } else {
        for (int i = tid; i < (past + rows) * size; i += kInThreads) {
            const int r = r0 - past + i / size, c = c0 + i % size;
            raw[i] = r >= 0 ? lm_sum_batch(a.in, r, c) : past_row(r, c);
        }
    }
    __syncthreads();
    /* a thread keeps to its channels, so that their taps stay in registers */
    constexpr int kRegTaps = 4;
    for (int d = tid; d < size; d += kInThreads) {
        const float *w = a.conv + (size_t)(c0 + d) * a.taps;
        float wr[kRegTaps];
        if (a.taps <= kRegTaps) {
#pragma unroll
            for (int j = 0; j < kRegTaps; j++) wr[j] = j < a.taps ? __ldg(w + j) : 0.0f;
        }
        for (int r = 0; r < rows; r++) {
            float v = 0.0f;
            if (a.taps <= kRegTaps) {
#pragma unroll
                for (int j = 0; j < kRegTaps; j++)
                    if (j < a.taps) v = fmaf(wr[j], raw[(r + j) * size + d], v);
            } else {
                for (int j = 0; j < a.taps; j++) v = fmaf(__ldg(w + j), raw[(r + j) * size + d], v);
            }
            out[(size_t)r * ld_out + d] = silu(v);
        }
    }
}

/* grid = (row tiles, kv_heads + heads + 1): q and k of a key head, v of a value head, or (last)
 * step sizes and decays. The q and k CTAs also leave the inner products of the scan's groups. */
__global__ void __launch_bounds__(kInThreads) lm_delta_inputs_kernel(const LmDelta a, int M) {
    extern __shared__ __align__(16) float in_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int r0 = blockIdx.x * kInRows, rows = M - r0 < kInRows ? M - r0 : kInRows;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, G = a.kv_heads, H = a.heads;
    const int nqk = G * a.dim, ch = 2 * nqk + H * a.vdim, unit = blockIdx.y;
    if (unit == G + H) {
        for (int i = tid; i < rows * H; i += kInThreads) {
            const int r = r0 + i / H, h = i % H;
            const int cb = ch + H * a.vdim;           /* columns: q, k, v, gate, b, a */
            a.beta[(size_t)r * H + h] = 1.0f / (1.0f + expf(-lm_sum(a.in, r, cb + h)));
            a.decays[(size_t)r * H + h] = expf(-__ldg(a.decay + h) * softplus(lm_sum(a.in, r, cb + H + h) + __ldg(a.dt_bias + h)));
        }
        return;
    }
    const int pos0 = a.dyn->pos;
    const float *tail = lm_state(a.tail, a.dyn);
    if (unit >= G) {
        const int head = unit - G;
        conv_rows(a, in_smem, a.v + (size_t)r0 * H * a.vdim + head * a.vdim, H * a.vdim, 2 * nqk + head * a.vdim, a.vdim, r0, rows, tail, ch,
                  pos0);
        return;
    }
    const int dim = a.dim;
    float *qk = in_smem, *raw = qk + 2 * kInRows * dim;         /* [q, k][kInRows][dim], room for the raw rows */
    for (int kind = 0; kind < 2; kind++) {
        float *out = qk + kind * kInRows * dim, *dst = kind == 0 ? a.q : a.k;
        conv_rows(a, raw, out, dim, kind * nqk + unit * dim, dim, r0, rows, tail, ch, pos0);
        __syncthreads();
        const float post = kind == 0 ? 1.0f / sqrtf((float)dim) : 1.0f;
        for (int r = warp; r < kInRows; r += kInThreads / 32) {
            float s = 0.0f;
            if (r < rows)
                for (int d = lane; d < dim; d += 32) s += out[r * dim + d] * out[r * dim + d];
            s = vb_warp_sum(s);
            const float f = 1.0f / sqrtf(s + 1e-6f) * post;
            for (int d = lane; d < dim; d += 32) {
                const float v = r < rows ? out[r * dim + d] * f : 0.0f;
                out[r * dim + d] = v;
                if (r < rows) dst[(size_t)(r0 + r) * nqk + unit * dim + d] = v;
            }
        }
        __syncthreads();
    }
    /* inner products inside a group of kScGroup tokens: k_t . k_j and q_t . k_j */
    const float *Q = qk, *K = qk + kInRows * dim;
    for (int i = warp; i < kInRows / kScGroup * kGramRow; i += kInThreads / 32) {
        const int j = i % kScGroup, t = i / kScGroup % kScGroup, isq = i / (kScGroup * kScGroup) % 2, grp = i / kGramRow;
        float s = 0.0f;
        if (j <= t) {
            const float *x = (isq ? Q : K) + (grp * kScGroup + t) * dim, *y = K + (grp * kScGroup + j) * dim;
            for (int d = lane; d < dim; d += 32) s = fmaf(x[d], y[d], s);
        }
        s = vb_warp_sum(s);
        if (lane == 0) a.gram[((size_t)(r0 / kScGroup + grp) * G + unit) * kGramRow + isq * kScGroup * kScGroup + t * kScGroup + j] = s;
    }
}

/* ------------------------------------------------------------------ the recurrence */
constexpr int kScCols = 16, kScTok = 16, kScGroups = kScTok / kScGroup, kScBufs = 3;

/* two fp32 lanes per instruction */
VB_DEVINL uint64_t f2_pack(float lo, float hi) {
    uint64_t r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r) : "f"(lo), "f"(hi));
    return r;
}
VB_DEVINL float f2_sum(uint64_t v) {
    float lo, hi;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(lo), "=f"(hi) : "l"(v));
    return lo + hi;
}
VB_DEVINL uint64_t f2_fma(uint64_t a, uint64_t b, uint64_t c) {
    uint64_t r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r) : "l"(a), "l"(b), "l"(c));
    return r;
}
VB_DEVINL uint64_t f2_add(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("add.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
VB_DEVINL uint64_t f2_mul(uint64_t a, uint64_t b) {
    uint64_t r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r) : "l"(a), "l"(b));
    return r;
}
VB_DEVINL void cp_async4(void *smem, const void *gmem) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(vb_smem_u32(smem)), "l"(gmem) : "memory");
}

/* Coefficients of one group of four tokens for one head. With c_t the product of the decays up to
 * token t of the group, d_tj that of the tokens after j up to t, and S the state before the group,
 *   u_t = beta_t v_t - beta_t c_t (S^T k_t) - sum_{j<t} beta_t d_tj (k_t . k_j) u_j
 *   o_t = c_t (S^T q_t) + sum_{j<=t} d_tj (q_t . k_j) u_j
 *   S  <- c_3 S + sum_j d_3j k_j u_j^T
 * which is the recurrence, token for token, with the four predictions taken from one S. */
struct __align__(16) ScanCoef {
    float beta[4], e[4];        /* beta_t; -beta_t c_t */
    float u[8];                 /* -beta_t d_tj (k_t . k_j) for (1,0) (2,0) (2,1) (3,0) (3,1) (3,2) */
    float s[4];                 /* d_3j */
    float o[4][4];              /* d_tj (q_t . k_j), zero for j > t */
    float c[4];                 /* c_t */
};

/* One buffer of the scan's inputs: kScTok tokens of k, q (padded to DP rows), the CTA's columns of v, step
 * sizes, decays and inner products, and the coefficients made of them. */
template <int DP>
struct __align__(16) ScanBuf {
    float k[kScTok][DP], q[kScTok][DP], v[kScTok][kScCols], gram[kScGroups][kGramRow], beta[kScTok], g[kScTok];
    ScanCoef coef[kScGroups];
};

/* grid = (value column tiles, heads). All warps but the last hold S: LPC lanes per column, each with
 * NR rows in groups of four (lane rg takes groups rg, rg + LPC, ...). Four tokens at a time: their
 * eight inner products with S (S^T k_t, S^T q_t) are independent and are summed over the lanes in
 * one halving butterfly, the rest is scalars. The last warp copies the inputs of the next blocks
 * of kScTok tokens (bulk copies where rows start on 16-byte boundaries) and works out their
 * coefficients. */
template <int LPC, int NR>
__global__ void __launch_bounds__(kScCols * LPC + 32) lm_delta_scan_kernel(const LmDelta a, int M) {
    static_assert(kScGroup == 4 && LPC >= 8, "the butterfly spreads eight values over at least eight lanes");
    constexpr int DP = LPC * NR, kCompute = kScCols * LPC, kThreads = kCompute + 32, NG = NR / 4;
    extern __shared__ __align__(16) unsigned char scan_smem[];
    __shared__ uint64_t full[kScBufs];
    __shared__ volatile int gave_up;
    ScanBuf<DP> *buf = reinterpret_cast<ScanBuf<DP> *>(scan_smem);
    pdl_launch_dependents();
    const int tid = threadIdx.x, lane = tid & 31, h = blockIdx.y, kv = h / (a.heads / a.kv_heads);
    const int c0 = blockIdx.x * kScCols;
    const int nqk = a.kv_heads * a.dim, nv = a.heads * a.vdim, n_blocks = (M + kScTok - 1) / kScTok;
    const bool bulk = ((a.dim | a.vdim) & 3) == 0;
    /* rows and columns beyond the sizes stay zero in every buffer */
    for (int i = tid; i < (int)(kScBufs * sizeof(ScanBuf<DP>) / 4); i += kThreads) reinterpret_cast<float *>(scan_smem)[i] = 0.0f;
    if (tid == 0) {
        for (int i = 0; i < kScBufs; i++) vb_mbar_init(&full[i], 1);
        gave_up = 0;
        vb_mbar_init_fence();
    }
    asm volatile("fence.proxy.async.shared::cta;" ::: "memory");      /* the zeros come before the copies */
    pdl_wait();
    __syncthreads();

    if (tid >= kCompute) {
        /* ---- inputs and coefficients ---- */
        const int cols = a.vdim - c0 < kScCols ? a.vdim - c0 : kScCols;
        auto request = [&](int blk) {
            if (blk < n_blocks && !gave_up) {
                const int b = blk % kScBufs;
                ScanBuf<DP> &d = buf[b];
                const int t0 = blk * kScTok, nt = M - t0 < kScTok ? M - t0 : kScTok, groups = (nt + kScGroup - 1) / kScGroup;
                const float *gram = a.gram + ((size_t)(t0 / kScGroup) * a.kv_heads + kv) * kGramRow;
                if (lane < nt) {
                    cp_async4(&d.beta[lane], a.beta + (size_t)(t0 + lane) * a.heads + h);
                    cp_async4(&d.g[lane], a.decays + (size_t)(t0 + lane) * a.heads + h);
                }
                if (bulk) {
                    if (lane == 0) vb_mbar_arrive_expect_tx(&full[b], (uint32_t)(4 * (nt * (2 * a.dim + cols) + groups * kGramRow)));
                    __syncwarp();
                    const int t = lane & 15;
                    const size_t at = (size_t)(t0 + t) * nqk + kv * a.dim;
                    if (t < nt) vb_bulk_g2s(lane < 16 ? d.k[t] : d.q[t], (lane < 16 ? a.k : a.q) + at, (uint32_t)a.dim * 4u, &full[b]);
                    if (lane < nt) vb_bulk_g2s(d.v[lane], a.v + (size_t)(t0 + lane) * nv + h * a.vdim + c0, (uint32_t)cols * 4u, &full[b]);
                    if (lane < groups) vb_bulk_g2s(d.gram[lane], gram + (size_t)lane * a.kv_heads * kGramRow, kGramRow * 4u, &full[b]);
                } else {
                    for (int t = 0; t < nt; t++) {
                        const size_t at = (size_t)(t0 + t) * nqk + kv * a.dim;
                        for (int i = lane; i < a.dim; i += 32) { cp_async4(&d.k[t][i], a.k + at + i); cp_async4(&d.q[t][i], a.q + at + i); }
                        if (lane < cols) cp_async4(&d.v[t][lane], a.v + (size_t)(t0 + t) * nv + h * a.vdim + c0 + lane);
                    }
                    for (int i = lane; i < groups * kGramRow; i += 32)
                        cp_async4(&d.gram[i / kGramRow][i % kGramRow], gram + (size_t)(i / kGramRow) * a.kv_heads * kGramRow + i % kGramRow);
                }
            }
            asm volatile("cp.async.commit_group;" ::: "memory");
        };
        auto arrived = [&](int blk) {                     /* everything requested for block blk has landed */
            asm volatile("cp.async.wait_group 1;" ::: "memory");
            if (bulk && blk < n_blocks && !vb_mbar_wait(&full[blk % kScBufs], (uint32_t)(blk / kScBufs) & 1u, &gave_up)) {
                atomicCAS(a.status, 0, 51);
                gave_up = 1;
            }
            __syncwarp();
        };
        auto coefficients = [&](int blk) {                /* one lane per group; tokens beyond the end change nothing */
            if (blk >= n_blocks || lane >= kScGroups) return;
            ScanBuf<DP> &d = buf[blk % kScBufs];
            const int nt = M - blk * kScTok, tg = lane * kScGroup;
            ScanCoef &x = d.coef[lane];
            float g[4], b[4], c = 1.0f;
#pragma unroll
            for (int t = 0; t < 4; t++) {
                g[t] = tg + t < nt ? d.g[tg + t] : 1.0f;
                b[t] = tg + t < nt ? d.beta[tg + t] : 0.0f;
            }
            int n = 0;
#pragma unroll
            for (int t = 0; t < 4; t++) {
                c *= g[t];
                x.beta[t] = b[t];
                x.e[t] = -b[t] * c;
                x.c[t] = c;
                float dt[4] = {0.0f, 0.0f, 0.0f, 0.0f}, p = 1.0f;
#pragma unroll
                for (int j = 3; j >= 0; j--) {
                    if (j > t) { x.o[t][j] = 0.0f; continue; }
                    dt[j] = p;
                    x.o[t][j] = tg + t < nt ? p * d.gram[lane][kScGroup * kScGroup + t * 4 + j] : 0.0f;
                    if (t == 3) x.s[j] = p;
                    p *= g[j];
                }
#pragma unroll
                for (int j = 0; j < t; j++) x.u[n++] = tg + t < nt ? -b[t] * dt[j] * d.gram[lane][t * 4 + j] : 0.0f;
            }
        };
        auto clear_tail = [&](int blk) {                  /* tokens beyond the end: no stale k, q, v in a used group */
            if (blk != n_blocks - 1) return;
            ScanBuf<DP> &d = buf[blk % kScBufs];
            const int nt = M - blk * kScTok, ne = (nt + kScGroup - 1) / kScGroup * kScGroup;
            for (int t = nt; t < ne; t++) {
                for (int i = lane; i < DP; i += 32) d.k[t][i] = d.q[t][i] = 0.0f;
                if (lane < kScCols) d.v[t][lane] = 0.0f;
            }
        };
        request(0);
        request(1);
        arrived(0);
        coefficients(0);
        clear_tail(0);
        __syncthreads();                                  /* block 0 is ready */
        for (int blk = 0; blk < n_blocks; blk++) {
            request(blk + 2);
            arrived(blk + 1);
            coefficients(blk + 1);
            clear_tail(blk + 1);
            __syncthreads();                              /* block blk is done with, blk + 1 is ready */
        }
        return;
    }

    const int rg = tid % LPC, cl = tid / LPC, c = c0 + cl;
    const bool live = c < a.vdim;
    float *S = lm_state(a.s, a.dyn) + (size_t)h * a.dim * a.vdim;
    uint64_t s[NR / 2];
    const bool fresh = a.dyn->pos == 0;
#pragma unroll
    for (int i = 0; i < NG; i++) {
        float x[4];
#pragma unroll
        for (int j = 0; j < 4; j++) {
            const int r = (i * LPC + rg) * 4 + j;
            x[j] = (!fresh && live && r < a.dim) ? S[(size_t)r * a.vdim + c] : 0.0f;
        }
        s[2 * i] = f2_pack(x[0], x[1]);
        s[2 * i + 1] = f2_pack(x[2], x[3]);
    }
    auto load = [&](uint64_t (&x)[NR / 2], const float *row) {
#pragma unroll
        for (int i = 0; i < NG; i++) {
            const ulonglong2 y = *reinterpret_cast<const ulonglong2 *>(row + (i * LPC + rg) * 4);
            x[2 * i] = y.x;
            x[2 * i + 1] = y.y;
        }
    };
    auto dot = [&](const uint64_t (&x)[NR / 2]) {
        uint64_t e0 = 0, e1 = 0;
#pragma unroll
        for (int i = 0; i < NR / 2; i += 2) {
            e0 = f2_fma(s[i], x[i], e0);
            e1 = f2_fma(s[i + 1], x[i + 1], e1);
        }
        return f2_sum(f2_add(e0, e1));
    };
    /* after the butterfly lane rg holds value rg / (LPC / 8): 0 .. 3 are S^T k_t, 4 .. 7 are S^T q_t */
    constexpr int kShare = LPC / 8;
    const int mine = rg / kShare, lane0 = lane & ~(LPC - 1), ot = mine & 3;
    const bool writes = live && mine >= 4 && rg % kShare == 0;
    float *out = a.o + h * a.vdim + c;
    __syncthreads();                                      /* block 0 is ready */
    for (int blk = 0; blk < n_blocks; blk++) {
        const ScanBuf<DP> &in = buf[blk % kScBufs];
        const int t0 = blk * kScTok, nt = M - t0 < kScTok ? M - t0 : kScTok;
        /* already complete: taken here too, so that this thread sees what the copies wrote */
        if (bulk && !vb_mbar_wait(&full[blk % kScBufs], (uint32_t)(blk / kScBufs) & 1u, &gave_up)) gave_up = 1;
        __syncwarp();
#pragma unroll 1
        for (int tg = 0; tg < nt; tg += kScGroup) {
            const ScanCoef &x = in.coef[tg / kScGroup];
            uint64_t k[4][NR / 2];
            float y[8];
#pragma unroll
            for (int t = 0; t < 4; t++) {
                uint64_t qt[NR / 2];
                load(k[t], in.k[tg + t]);
                load(qt, in.q[tg + t]);
                y[t] = dot(k[t]);
                y[4 + t] = dot(qt);
            }
            const float4 beta = *reinterpret_cast<const float4 *>(x.beta), ec = *reinterpret_cast<const float4 *>(x.e),
                         u0 = *reinterpret_cast<const float4 *>(x.u), u1 = *reinterpret_cast<const float4 *>(x.u + 4),
                         sc = *reinterpret_cast<const float4 *>(x.s), oc = *reinterpret_cast<const float4 *>(x.o[ot]);
            const float oe = x.c[ot], c3 = x.c[3];
            const float v0 = beta.x * in.v[tg][cl], v1 = beta.y * in.v[tg + 1][cl], v2 = beta.z * in.v[tg + 2][cl], v3 = beta.w * in.v[tg + 3][cl];
            /* eight sums over the LPC lanes */
#pragma unroll
            for (int n = 4, off = LPC / 2; n >= 1; n >>= 1, off >>= 1) {
                const bool up = (rg & off) != 0;
#pragma unroll
                for (int i = 0; i < n; i++) {
                    const float send = up ? y[i] : y[i + n], keep = up ? y[i + n] : y[i];
                    y[i] = keep + __shfl_xor_sync(0xffffffffu, send, off);
                }
            }
#pragma unroll
            for (int off = kShare / 2; off >= 1; off >>= 1) y[0] += __shfl_xor_sync(0xffffffffu, y[0], off);
            const float e0 = __shfl_sync(0xffffffffu, y[0], lane0), e1 = __shfl_sync(0xffffffffu, y[0], lane0 + kShare),
                        e2 = __shfl_sync(0xffffffffu, y[0], lane0 + 2 * kShare), e3 = __shfl_sync(0xffffffffu, y[0], lane0 + 3 * kShare);
            const uint64_t cc = f2_pack(c3, c3);
#pragma unroll
            for (int i = 0; i < NR / 2; i++) s[i] = f2_mul(s[i], cc);
            const float w0 = fmaf(ec.x, e0, v0);
            const float w1 = fmaf(u0.x, w0, fmaf(ec.y, e1, v1));
            const float w2 = fmaf(u0.z, w1, fmaf(u0.y, w0, fmaf(ec.z, e2, v2)));
            const float w3 = fmaf(u1.y, w2, fmaf(u1.x, w1, fmaf(u0.w, w0, fmaf(ec.w, e3, v3))));
            const uint64_t d0 = f2_pack(sc.x * w0, sc.x * w0), d1 = f2_pack(sc.y * w1, sc.y * w1), d2 = f2_pack(sc.z * w2, sc.z * w2),
                           d3 = f2_pack(sc.w * w3, sc.w * w3);
#pragma unroll
            for (int i = 0; i < NR / 2; i++) s[i] = f2_fma(k[3][i], d3, f2_fma(k[2][i], d2, f2_fma(k[1][i], d1, f2_fma(k[0][i], d0, s[i]))));
            const float o = fmaf(oc.w, w3, fmaf(oc.z, w2, fmaf(oc.y, w1, fmaf(oc.x, w0, oe * y[0]))));
            if (writes && tg + ot < nt) out[(size_t)(t0 + tg + ot) * nv] = o;
        }
        __syncthreads();                                  /* block blk is done with, blk + 1 is ready */
    }
#pragma unroll
    for (int i = 0; i < NR / 2; i++) {
        float x[2];
        asm("mov.b64 {%0, %1}, %2;" : "=f"(x[0]), "=f"(x[1]) : "l"(s[i]));
#pragma unroll
        for (int j = 0; j < 2; j++) {
            const int r = ((i / 2) * LPC + rg) * 4 + (i & 1) * 2 + j;
            if (live && r < a.dim) S[(size_t)r * a.vdim + c] = x[j];
        }
    }
}

template <int LPC, int NR>
int launch_scan(const LmDelta &a, int M, cudaStream_t st) {
    constexpr size_t smem = kScBufs * sizeof(ScanBuf<LPC * NR>);
    static_assert(smem <= 220 * 1024, "over what a CTA may use");
    static bool attr = false;
    if (!attr) {
        if (cudaFuncSetAttribute(lm_delta_scan_kernel<LPC, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        attr = true;
    }
    /* A plain launch: started early, under the tail of the kernel before it, the CTAs would crowd onto the first
     * SMs that have room, and this kernel's time is that of its most crowded SM. */
    lm_delta_scan_kernel<LPC, NR><<<dim3((a.vdim + kScCols - 1) / kScCols, a.heads), kScCols * LPC + 32, smem, st>>>(a, M);
    return ok(cudaGetLastError());
}

/* ------------------------------------------------------------------ head norm, gate, convolution memory */
constexpr int kGtThreads = 256;

/* grid = rows; a warp per head. The CTAs of the last `taps` rows also save their raw convolution
 * inputs (everything that reads the memory's old content ran in earlier launches). */
__global__ void __launch_bounds__(kGtThreads) lm_delta_gate_kernel(const LmDelta a, int M) {
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int nv = a.heads * a.vdim, ch = 2 * a.kv_heads * a.dim + nv;
    for (int h = warp; h < a.heads; h += kGtThreads / 32) {
        const float *o = a.o + (size_t)m * nv + h * a.vdim;
        float s = 0.0f;
        for (int d = lane; d < a.vdim; d += 32) s += o[d] * o[d];
        const float r = 1.0f / sqrtf(vb_warp_sum(s) / (float)a.vdim + a.eps);
        for (int d = lane; d < a.vdim; d += 32)
            lm_put(a.out, m, h * a.vdim + d, o[d] * r * __ldg(a.norm + d) * silu(lm_sum(a.in, m, ch + h * a.vdim + d)));
    }
    if (m >= M - a.taps) {
        float *tail = lm_state(a.tail, a.dyn) + (size_t)((a.dyn->pos + m) % a.taps) * ch;
        for (int c = tid; c < ch; c += kGtThreads) tail[c] = lm_sum(a.in, m, c);
    }
}

/* ------------------------------------------------------------------ one token */
constexpr int kStThreads = 512, kStWarps = 16, kStCols = 32, kStTaps = 4;

/* grid = (value column slices, heads), the slices of a head form a cluster. Warp w holds rows
 * w, w + 16, ... of S, a lane one column. The memory row of the convolution that is written
 * (position p, row p % taps) is none of those that other CTAs read (p - 1 ... p - taps + 1). */
template <int NR>
__global__ void __launch_bounds__(kStThreads) lm_delta_step_kernel(const LmDelta a) {
    __shared__ float qs[kStWarps * NR], ks[kStWarps * NR], vs[kStCols], red[2][kStWarps], part[2][kStWarps][kStCols], scal[2], ssq;
    namespace cg = cooperative_groups;
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int h = blockIdx.y, group = a.heads / a.kv_heads, kv = h / group, H = a.heads;
    const int col0 = blockIdx.x * kStCols, c = col0 + lane;
    const bool live = c < a.vdim;
    const int pos = a.dyn->pos, nqk = a.kv_heads * a.dim, ch = 2 * nqk + H * a.vdim;
    float *S = lm_state(a.s, a.dyn) + (size_t)h * a.dim * a.vdim;
    float *tail = lm_state(a.tail, a.dyn);

    /* the state is requested first: it is the long way */
    float s[NR];
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int r = warp + kStWarps * i;
        s[i] = (pos > 0 && live && r < a.dim) ? __ldcg(S + (size_t)r * a.vdim + c) : 0.0f;
    }
    float gate = 0.0f;
    if (warp == 0 && live) gate = lm_sum_batch(a.in, 0, ch + h * a.vdim + c);
    if (warp == 1 && lane < 2) {
        const float x = lm_sum_batch(a.in, 0, ch + H * a.vdim + lane * H + h);
        scal[lane] = lane == 0 ? 1.0f / (1.0f + expf(-x)) : expf(-__ldg(a.decay + h) * softplus(x + __ldg(a.dt_bias + h)));
    }
    /* convolution of this head's q and k and of the slice's v */
    const int ncols = a.vdim - col0 < kStCols ? a.vdim - col0 : kStCols;
    float sq = 0.0f, sk = 0.0f;
    for (int i = tid; i < 2 * a.dim + ncols; i += kStThreads) {
        const int kind = i < a.dim ? 0 : i < 2 * a.dim ? 1 : 2;
        const int chan = kind == 0 ? kv * a.dim + i : kind == 1 ? nqk + kv * a.dim + i - a.dim : 2 * nqk + h * a.vdim + col0 + i - 2 * a.dim;
        const float raw = lm_sum_batch(a.in, 0, chan);
        const float *w = a.conv + (size_t)chan * a.taps;
        float v = 0.0f;
        for (int j0 = 0; j0 < a.taps - 1; j0 += kStTaps) {
            float x[kStTaps], wj[kStTaps];              /* requested together, unconditionally */
#pragma unroll
            for (int u = 0; u < kStTaps; u++) {
                const int j = j0 + u < a.taps - 1 ? j0 + u : j0, p = pos - (a.taps - 1) + j;
                x[u] = __ldcg(tail + (size_t)((p + a.taps) % a.taps) * ch + chan);
                wj[u] = __ldg(w + j);
            }
#pragma unroll
            for (int u = 0; u < kStTaps; u++)
                if (j0 + u < a.taps - 1 && pos - (a.taps - 1) + j0 + u >= 0) v = fmaf(wj[u], x[u], v);
        }
        v = silu(fmaf(__ldg(w + a.taps - 1), raw, v));
        if (kind == 2 || (blockIdx.x == 0 && h % group == 0)) tail[(size_t)(pos % a.taps) * ch + chan] = raw;
        if (kind == 0) { qs[i] = v; sq += v * v; }
        else if (kind == 1) { ks[i - a.dim] = v; sk += v * v; }
        else vs[i - 2 * a.dim] = v;
    }
    for (int i = a.dim + tid; i < kStWarps * NR; i += kStThreads) qs[i] = ks[i] = 0.0f;
    sq = vb_warp_sum(sq);
    sk = vb_warp_sum(sk);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < kStWarps; w++) { sq += red[0][w]; sk += red[1][w]; }
    const float fq = 1.0f / sqrtf(sq + 1e-6f) / sqrtf((float)a.dim), fk = 1.0f / sqrtf(sk + 1e-6f);
    const float beta = scal[0], g = scal[1];
    float e = 0.0f;
#pragma unroll
    for (int i = 0; i < NR; i++) {
        s[i] *= g;
        e = fmaf(s[i], ks[warp + kStWarps * i] * fk, e);
    }
    part[0][warp][lane] = e;
    __syncthreads();
    e = 0.0f;
#pragma unroll
    for (int w = 0; w < kStWarps; w++) e += part[0][w][lane];
    const float u = live ? beta * (vs[lane] - e) : 0.0f;
    float o = 0.0f;
#pragma unroll
    for (int i = 0; i < NR; i++) {
        s[i] = fmaf(ks[warp + kStWarps * i] * fk, u, s[i]);
        o = fmaf(s[i], qs[warp + kStWarps * i] * fq, o);
    }
    part[1][warp][lane] = o;
#pragma unroll
    for (int i = 0; i < NR; i++) {
        const int r = warp + kStWarps * i;
        if (live && r < a.dim) S[(size_t)r * a.vdim + c] = s[i];
    }
    __syncthreads();
    if (warp == 0) {
        o = 0.0f;
#pragma unroll
        for (int w = 0; w < kStWarps; w++) o += part[1][w][lane];
        const float t = vb_warp_sum(live ? o * o : 0.0f);
        if (lane == 0) ssq = t;
    }
    /* the head's norm spans the cluster's slices */
    cg::cluster_group cluster = cg::this_cluster();
    cluster.sync();
    if (warp == 0) {
        float t = 0.0f;
        for (unsigned r = 0; r < cluster.num_blocks(); r++) t += *cluster.map_shared_rank(&ssq, r);
        const float rn = 1.0f / sqrtf(t / (float)a.vdim + a.eps);
        if (live) lm_put(a.out, 0, h * a.vdim + c, o * rn * __ldg(a.norm + c) * silu(gate));
    }
    cluster.sync();                                   /* nobody leaves while its sum may still be read */
}

template <int NR>
int launch_step(const LmDelta &a, cudaStream_t st) {
    cudaLaunchConfig_t cfg = {};
    const unsigned slices = (unsigned)(a.vdim + kStCols - 1) / kStCols;
    cfg.gridDim = dim3(slices, a.heads); cfg.blockDim = dim3(kStThreads); cfg.stream = st;
    cudaLaunchAttribute at[2];
    at[0].id = cudaLaunchAttributeClusterDimension;
    at[0].val.clusterDim.x = slices; at[0].val.clusterDim.y = 1; at[0].val.clusterDim.z = 1;
    at[1].id = cudaLaunchAttributeProgrammaticStreamSerialization;
    at[1].val.programmaticStreamSerializationAllowed = 1;
    cfg.attrs = at;
    static const bool no_pdl = getenv("VB200_NO_PDL") != nullptr;
    cfg.numAttrs = no_pdl ? 1 : 2;
    return ok(cudaLaunchKernelEx(&cfg, lm_delta_step_kernel<NR>, a));
}

} // namespace

int lm_delta_channels(int heads, int kv_heads, int dim, int vdim) { return 2 * kv_heads * dim + heads * vdim; }
bool lm_delta_supported(int dim, int vdim) { return dim >= 1 && dim <= 256 && vdim >= 1; }

int lm_delta_inputs(const LmDelta &a, int M, cudaStream_t st) {
    const size_t raw = kInRows + a.taps - 1, qk = (raw + 2 * kInRows) * a.dim, v = raw * a.vdim;
    const size_t smem = sizeof(float) * (qk > v ? qk : v);
    if (smem > 200 * 1024) return -1;
    static size_t set = 48 * 1024;
    if (smem > set) {
        if (cudaFuncSetAttribute(lm_delta_inputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        set = smem;
    }
    return ok(launch_pdl(lm_delta_inputs_kernel, dim3((M + kInRows - 1) / kInRows, a.kv_heads + a.heads + 1), dim3(kInThreads), smem,
                         st, a, M));
}

int lm_delta_scan(const LmDelta &a, int M, cudaStream_t st) {
    if (a.dim <= 32) return launch_scan<8, 4>(a, M, st);
    if (a.dim <= 64) return launch_scan<8, 8>(a, M, st);
    if (a.dim <= 128) return launch_scan<8, 16>(a, M, st);
    if (a.dim <= 256) return launch_scan<16, 16>(a, M, st);
    return -1;
}

int lm_delta_gate(const LmDelta &a, int M, cudaStream_t st) {
    return ok(launch_pdl(lm_delta_gate_kernel, dim3(M), dim3(kGtThreads), 0, st, a, M));
}

bool lm_delta_step_ok(const LmDelta &a) { return a.dim <= 256 && a.vdim <= 8 * kStCols; }

int lm_delta_step(const LmDelta &a, cudaStream_t st) {
    if (a.dim <= 64) return launch_step<4>(a, st);
    if (a.dim <= 128) return launch_step<8>(a, st);
    return launch_step<16>(a, st);
}

} // namespace vb
