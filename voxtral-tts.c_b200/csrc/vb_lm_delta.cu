/*
 * vb_lm_delta.cu - decoder language models: gated delta-rule mixer.
 *
 *   q, k, v = silu(short causal convolution of the projections), q and k made unit vectors
 *   S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q        (per head, fp32)
 *   out = rmsnorm(o) * silu(gate)
 *
 *   lm_delta_inputs  convolution, unit norms, step sizes beta, decays: 16 rows per CTA
 *   lm_delta_scan    the recurrence token by token, in fp32; columns of S are independent, so a CTA owns
 *                    16 of a head's value columns, S in registers, eight lanes per column
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
constexpr int kInThreads = 128, kInRows = 16;

/* grid = (row tiles, 2 * kv_heads + heads + 1): one head of q, k or v per CTA; the last column of
 * CTAs works out step sizes and decays. */
__global__ void __launch_bounds__(kInThreads) lm_delta_inputs_kernel(const LmDelta a, int M) {
    extern __shared__ __align__(16) float in_smem[];
    pdl_launch_dependents();
    pdl_wait();
    const int r0 = blockIdx.x * kInRows, rows = M - r0 < kInRows ? M - r0 : kInRows;
    const int tid = threadIdx.x, G = a.kv_heads, H = a.heads;
    const int nqk = G * a.dim, ch = 2 * nqk + H * a.vdim;
    int unit = blockIdx.y;
    if (unit == 2 * G + H) {
        for (int i = tid; i < rows * H; i += kInThreads) {
            const int r = r0 + i / H, h = i % H;
            const int cb = ch + H * a.vdim;           /* columns: q, k, v, gate, b, a */
            a.beta[(size_t)r * H + h] = 1.0f / (1.0f + expf(-lm_sum(a.in, r, cb + h)));
            a.decays[(size_t)r * H + h] = expf(-__ldg(a.decay + h) * softplus(lm_sum(a.in, r, cb + H + h) + __ldg(a.dt_bias + h)));
        }
        return;
    }
    const int kind = unit < G ? 0 : unit < 2 * G ? 1 : 2;     /* q, k, v */
    const int head = kind == 2 ? unit - 2 * G : unit % G;
    const int size = kind == 2 ? a.vdim : a.dim;
    const int c0 = kind == 2 ? 2 * nqk + head * a.vdim : kind * nqk + head * a.dim;   /* first channel */
    const int past = a.taps - 1;
    float *raw = in_smem, *out = raw + (kInRows + past) * size;      /* [past + rows][size], [rows][size] */
    const int pos0 = a.dyn->pos;
    const float *tail = lm_state(a.tail, a.dyn);
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
            v = silu(v);
            if (kind == 2) a.v[(size_t)(r0 + r) * H * a.vdim + head * a.vdim + d] = v;
            else out[r * size + d] = v;
        }
    }
    if (kind == 2) return;
    __syncthreads();
    const int warp = tid >> 5, lane = tid & 31;
    float *dst = kind == 0 ? a.q : a.k;
    const float post = kind == 0 ? 1.0f / sqrtf((float)a.dim) : 1.0f;
    for (int r = warp; r < rows; r += kInThreads / 32) {
        float s = 0.0f;
        for (int d = lane; d < size; d += 32) s += out[r * size + d] * out[r * size + d];
        s = vb_warp_sum(s);
        const float f = 1.0f / sqrtf(s + 1e-6f) * post;
        for (int d = lane; d < size; d += 32) dst[(size_t)(r0 + r) * nqk + head * a.dim + d] = out[r * size + d] * f;
    }
}

/* ------------------------------------------------------------------ the recurrence, token by token */
constexpr int kScCols = 16, kScTok = 16;

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
VB_DEVINL void cp_async16(void *smem, const void *gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(vb_smem_u32(smem)), "l"(gmem) : "memory");
}

/* One buffer of the scan's inputs: kScTok tokens of k, q (padded to DP rows), the CTA's columns of v, step
 * sizes and decays. */
template <int DP>
struct ScanBuf {
    float k[kScTok][DP], q[kScTok][DP], v[kScTok][kScCols], beta[kScTok], g[kScTok];
};

/* grid = (value column tiles, heads), LPC lanes per column, each with NR rows of S: groups of four
 * rows, lane rg takes groups rg, rg + LPC, ... Per token the read-out of the token before and the
 * prediction S^T k are taken from the same S, so that one pass and one round of shuffles serves
 * both; the decay is applied to the prediction and, while the sums travel, to S. The inputs of the
 * next kScTok tokens are copied while the current ones are worked on. */
template <int LPC, int NR>
__global__ void __launch_bounds__(kScCols * LPC) lm_delta_scan_kernel(const LmDelta a, int M) {
    constexpr int DP = LPC * NR, kThreads = kScCols * LPC, NG = NR / 4;
    extern __shared__ __align__(16) unsigned char scan_smem[];
    ScanBuf<DP> *buf = reinterpret_cast<ScanBuf<DP> *>(scan_smem);
    pdl_launch_dependents();
    const int tid = threadIdx.x, h = blockIdx.y, kv = h / (a.heads / a.kv_heads);
    const int rg = tid % LPC, cl = tid / LPC, c0 = blockIdx.x * kScCols, c = c0 + cl;
    const bool live = c < a.vdim;
    const int nqk = a.kv_heads * a.dim, nv = a.heads * a.vdim;
    /* rows and columns beyond the sizes stay zero in both buffers */
    for (int i = tid; i < (int)(2 * sizeof(ScanBuf<DP>) / 4); i += kThreads) reinterpret_cast<float *>(scan_smem)[i] = 0.0f;
    pdl_wait();
    __syncthreads();
    auto request = [&](int t0, int b) {
        const int nt = M - t0 < kScTok ? M - t0 : kScTok;
        if ((a.dim & 3) == 0) {
            const int per = a.dim / 4;
            for (int i = tid; i < nt * per; i += kThreads) {
                const int t = i / per, d = i % per * 4;
                const size_t at = (size_t)(t0 + t) * nqk + kv * a.dim + d;
                cp_async16(&buf[b].k[t][d], a.k + at);
                cp_async16(&buf[b].q[t][d], a.q + at);
            }
        } else {
            for (int i = tid; i < nt * a.dim; i += kThreads) {
                const int t = i / a.dim, d = i % a.dim;
                const size_t at = (size_t)(t0 + t) * nqk + kv * a.dim + d;
                cp_async4(&buf[b].k[t][d], a.k + at);
                cp_async4(&buf[b].q[t][d], a.q + at);
            }
        }
        for (int i = tid; i < nt * kScCols; i += kThreads) {
            const int t = i / kScCols, cc = i % kScCols;
            if (c0 + cc < a.vdim) cp_async4(&buf[b].v[t][cc], a.v + (size_t)(t0 + t) * nv + h * a.vdim + c0 + cc);
        }
        if (tid < nt) {
            cp_async4(&buf[b].beta[tid], a.beta + (size_t)(t0 + tid) * a.heads + h);
            cp_async4(&buf[b].g[tid], a.decays + (size_t)(t0 + tid) * a.heads + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    request(0, 0);

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
    float *out = a.o + h * a.vdim + c;
    uint64_t qp[NR / 2];                                  /* query of the token before */
#pragma unroll
    for (int i = 0; i < NR / 2; i++) qp[i] = 0;
    auto load = [&](uint64_t (&x)[NR / 2], const float *row) {
#pragma unroll
        for (int i = 0; i < NG; i++) {
            const ulonglong2 y = *reinterpret_cast<const ulonglong2 *>(row + (i * LPC + rg) * 4);
            x[2 * i] = y.x;
            x[2 * i + 1] = y.y;
        }
    };
    for (int t0 = 0, b = 0; t0 < M; t0 += kScTok, b ^= 1) {
        const int nt = M - t0 < kScTok ? M - t0 : kScTok;
        asm volatile("cp.async.wait_group 0;" ::: "memory");
        __syncthreads();                                  /* this buffer is complete, the other one is free */
        if (t0 + kScTok < M) request(t0 + kScTok, b ^ 1);
        const ScanBuf<DP> &in = buf[b];
        uint64_t k[NR / 2];
        load(k, in.k[0]);
        float g = in.g[0], beta = in.beta[0], v = in.v[0][cl];
#pragma unroll 2
        for (int t = 0; t < nt; t++) {
            uint64_t e0 = 0, e1 = 0, o0 = 0, o1 = 0;
#pragma unroll
            for (int i = 0; i < NR / 2; i += 2) {
                e0 = f2_fma(s[i], k[i], e0);
                e1 = f2_fma(s[i + 1], k[i + 1], e1);
                o0 = f2_fma(s[i], qp[i], o0);
                o1 = f2_fma(s[i + 1], qp[i + 1], o1);
            }
            float e = f2_sum(f2_add(e0, e1)), o = f2_sum(f2_add(o0, o1));
            /* independent of the reductions: the decayed S, the next token's inputs (the last one's again at the
             * end), this token's query */
            const int tn = t + 1 < nt ? t + 1 : t;
            const uint64_t g2 = f2_pack(g, g);
            const float bv = beta * v, bg = -beta * g;
            uint64_t kn[NR / 2];
            load(kn, in.k[tn]);
            g = in.g[tn]; beta = in.beta[tn]; v = in.v[tn][cl];
            load(qp, in.q[t]);
#pragma unroll
            for (int i = 0; i < NR / 2; i++) s[i] = f2_mul(s[i], g2);
#pragma unroll
            for (int x = 1; x < LPC; x <<= 1) {
                e += __shfl_xor_sync(0xffffffffu, e, x);
                o += __shfl_xor_sync(0xffffffffu, o, x);
            }
            const float u = fmaf(bg, e, bv);              /* beta (v - g S^T k) */
            const uint64_t u2 = f2_pack(u, u);
#pragma unroll
            for (int i = 0; i < NR / 2; i++) {
                s[i] = f2_fma(k[i], u2, s[i]);
                k[i] = kn[i];
            }
            if (rg == 0 && live && t0 + t > 0) out[(size_t)(t0 + t - 1) * nv] = o;
        }
    }
    uint64_t o0 = 0, o1 = 0;
#pragma unroll
    for (int i = 0; i < NR / 2; i += 2) {
        o0 = f2_fma(s[i], qp[i], o0);
        o1 = f2_fma(s[i + 1], qp[i + 1], o1);
    }
    float o = f2_sum(o0) + f2_sum(o1);
#pragma unroll
    for (int x = 1; x < LPC; x <<= 1) o += __shfl_xor_sync(0xffffffffu, o, x);
    if (rg == 0 && live) out[(size_t)(M - 1) * nv] = o;
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
    constexpr size_t smem = 2 * sizeof(ScanBuf<LPC * NR>);
    static bool attr = false;
    if (!attr) {
        if (cudaFuncSetAttribute(lm_delta_scan_kernel<LPC, NR>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        attr = true;
    }
    return ok(launch_pdl(lm_delta_scan_kernel<LPC, NR>, dim3((a.vdim + kScCols - 1) / kScCols, a.heads), dim3(kScCols * LPC), smem, st, a, M));
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
    const int size = a.dim > a.vdim ? a.dim : a.vdim;
    const size_t smem = sizeof(float) * (size_t)(2 * kInRows + a.taps - 1) * size;
    if (smem > 200 * 1024) return -1;
    static size_t set = 48 * 1024;
    if (smem > set) {
        if (cudaFuncSetAttribute(lm_delta_inputs_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        set = smem;
    }
    return ok(launch_pdl(lm_delta_inputs_kernel, dim3((M + kInRows - 1) / kInRows, 2 * a.kv_heads + a.heads + 1), dim3(kInThreads), smem,
                         st, a, M));
}

int lm_delta_scan(const LmDelta &a, int M, cudaStream_t st) {
    if (a.dim <= 32) return launch_scan<8, 4>(a, M, st);
    if (a.dim <= 64) return launch_scan<8, 8>(a, M, st);
    if (a.dim <= 128) return launch_scan<8, 16>(a, M, st);
    if (a.dim <= 256) return launch_scan<8, 32>(a, M, st);
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
