/*
 * vb_lm_kernels.cu - decoder language models: residual stream and norms, weight repacking, the
 * fp32 GEMM of the 32-bit mode, greedy choice of the next token.
 */
#include "vb_lm_kernels.cuh"

#include "vb_tc.cuh"

namespace vb {

namespace {

/* Sum over the CTA; `red` holds one float per warp and is a different array for successive calls. */
VB_DEVINL float cta_sum(float v, float *red) {
    v = vb_warp_sum(v);
    const int lane = threadIdx.x & 31, warps = (int)blockDim.x >> 5;
    if (lane == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    return vb_warp_sum(lane < warps ? red[lane] : 0.0f);
}

/* One row of the residual stream per CTA, held in registers: the sublayer's output (split-K
 * partials) is normalised or taken as it is, added to the stream, and the new row is normalised for
 * the next sublayer. Variances are means of squared deviations. A thread owns NV groups of VEC columns. */
template <int VEC, int NV>
__global__ void __launch_bounds__(1024) lm_residual_kernel(const LmResidual a) {
    __shared__ float red[4][32];
    constexpr int N = VEC * NV;
    pdl_launch_dependents();
    const int m = blockIdx.x, tid = threadIdx.x, W = a.width;
    const float inv_w = 1.0f / (float)W;
    auto col = [&](int i) { return (tid + i * (int)blockDim.x) * VEC; };
    /* the gains depend on nothing that runs before */
    float gp[N], gn[N];
#pragma unroll
    for (int i = 0; i < NV; i++)
#pragma unroll
        for (int j = 0; j < VEC; j++) {
            const int c = col(i) + j;
            gp[i * VEC + j] = a.join == LM_JOIN_NORMED && c < W ? __ldg(a.post_gain + c) : 0.0f;
            gn[i * VEC + j] = a.next == LM_NEXT_NORM && c < W ? __ldg(a.next_gain + c) : 0.0f;
        }
    pdl_wait();
    const int src = a.row_of ? a.row_of[m] : m;
    float x[N];
    const bool need0 = a.first || a.next == LM_NEXT_CONCAT;
    const uint16_t *e0 = need0 ? a.embed + (size_t)a.tokens[src] * W : nullptr;
    if (a.first) {
#pragma unroll
        for (int i = 0; i < NV; i++)
#pragma unroll
            for (int j = 0; j < VEC; j++) x[i * VEC + j] = col(i) < W ? __uint_as_float((uint32_t)e0[col(i) + j] << 16) : 0.0f;
    } else {
        float r[N];
        const bool add = a.join != LM_JOIN_REPLACE;
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = col(i);
            const bool in = c < W;
            if constexpr (VEC == 4) {
                const float4 rv = in && add ? __ldcg(reinterpret_cast<const float4 *>(a.x + (size_t)src * W + c)) : make_float4(0.f, 0.f, 0.f, 0.f);
                const float4 xv = in ? lm_sum4(a.part, src, c) : make_float4(0.f, 0.f, 0.f, 0.f);
                x[i * 4] = xv.x; x[i * 4 + 1] = xv.y; x[i * 4 + 2] = xv.z; x[i * 4 + 3] = xv.w;
                r[i * 4] = rv.x; r[i * 4 + 1] = rv.y; r[i * 4 + 2] = rv.z; r[i * 4 + 3] = rv.w;
            } else {
                r[i] = in && add ? a.x[(size_t)src * W + c] : 0.0f;
                x[i] = in ? lm_sum_batch(a.part, src, c) : 0.0f;
            }
        }
        for (int k = 0; k < a.mix.top; k++) {              /* the chosen experts, weighted */
            const float p = a.mix.weight[(size_t)src * a.mix.top + k];
            const float *y = a.mix.y + (size_t)a.mix.at[(size_t)src * a.mix.top + k] * a.mix.ld;
#pragma unroll
            for (int i = 0; i < NV; i++) {
                const int c = col(i);
                if (c >= W) continue;
                if constexpr (VEC == 4) {
                    const float4 v = vb_ldcg4(y + c);
                    x[i * 4] = fmaf(p, v.x, x[i * 4]); x[i * 4 + 1] = fmaf(p, v.y, x[i * 4 + 1]);
                    x[i * 4 + 2] = fmaf(p, v.z, x[i * 4 + 2]); x[i * 4 + 3] = fmaf(p, v.w, x[i * 4 + 3]);
                } else {
                    x[i] = fmaf(p, vb_ldcg(y + c), x[i]);
                }
            }
        }
        if (a.join == LM_JOIN_ADD) {
#pragma unroll
            for (int i = 0; i < N; i++) x[i] = r[i] + x[i];
        } else if (add) {
            float s = 0.0f;
#pragma unroll
            for (int i = 0; i < N; i++) s += x[i];
            const float mean = a.rms ? 0.0f : cta_sum(s, red[0]) * inv_w;
            s = 0.0f;
#pragma unroll
            for (int i = 0; i < N; i++) {
                x[i] = col(i / VEC) < W ? x[i] - mean : 0.0f;
                s += x[i] * x[i];
            }
            const float rstd = 1.0f / sqrtf(cta_sum(s, red[1]) * inv_w + a.eps);
#pragma unroll
            for (int i = 0; i < N; i++) x[i] = r[i] + x[i] * rstd * gp[i];      /* zero beyond the row */
        }
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int c = col(i);
        if (c >= W) continue;
#pragma unroll
        for (int t = 0; t < 2; t++) {
            float *dst = t ? a.tap : a.row_of ? nullptr : a.x;
            if (!dst) continue;
            dst += (size_t)m * W + c;
            if constexpr (VEC == 4) *reinterpret_cast<float4 *>(dst) = make_float4(x[i * 4], x[i * 4 + 1], x[i * 4 + 2], x[i * 4 + 3]);
            else *dst = x[i];
        }
    }
    auto put = [&](int c, const float *v) {
        if constexpr (VEC == 4) {
            const float q[4] = {v[0], v[1], v[2], v[3]};
            lm_put4(a.sink, m, c, q);
        } else {
            lm_put(a.sink, m, c, *v);
        }
    };
    if (a.next == LM_NEXT_NORM) {
        float s = 0.0f;
#pragma unroll
        for (int i = 0; i < N; i++) s += x[i];
        const float mean = a.rms ? 0.0f : cta_sum(s, red[2]) * inv_w;
        s = 0.0f;
#pragma unroll
        for (int i = 0; i < N; i++) {
            x[i] = col(i / VEC) < W ? x[i] - mean : 0.0f;
            s += x[i] * x[i];
        }
        const float rstd = 1.0f / sqrtf(cta_sum(s, red[3]) * inv_w + a.eps);
#pragma unroll
        for (int i = 0; i < N; i++) x[i] = x[i] * rstd * gn[i];
#pragma unroll
        for (int i = 0; i < NV; i++)
            if (col(i) < W) put(col(i), x + i * VEC);
    } else if (a.next == LM_NEXT_CONCAT) {
#pragma unroll
        for (int i = 0; i < NV; i++) {
            const int c = col(i);
            if (c >= W) continue;
            float e[VEC];
#pragma unroll
            for (int j = 0; j < VEC; j++) e[j] = __uint_as_float((uint32_t)e0[c + j] << 16);
            put(c, x + i * VEC);
            put(W + c, e);
        }
    }
}

__global__ void lm_pack_rows_kernel(uint16_t *dst, int Kp, int row0, int step, int col0, const uint16_t *src, int rows, int K) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)rows * K) return;
    const int r = (int)(i / K), c = (int)(i % K);
    dst[(size_t)(row0 + (long long)r * step) * Kp + col0 + c] = src[i];
}

__global__ void lm_widen_kernel(float *dst, const uint16_t *src, int n) {
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) dst[i] = __uint_as_float((uint32_t)src[i] << 16);
}

/* Sum of four hashed uniforms, about normal, scaled: weights of a benchmark model. */
__global__ void lm_fill_random_kernel(uint16_t *dst, size_t n, uint32_t seed, float mean, float scale) {
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= n) return;
    uint32_t h = (uint32_t)i * 2654435761u ^ (uint32_t)(i >> 32) * 40503u ^ seed;
    float s = 0.0f;
    for (int k = 0; k < 4; k++) {
        h ^= h >> 16; h *= 0x7feb352du; h ^= h >> 15; h *= 0x846ca68bu; h ^= h >> 16;
        s += (float)(h >> 8) * (1.0f / 16777216.0f) - 0.5f;
    }
    dst[i] = __bfloat16_as_ushort(__float2bfloat16_rn(mean + scale * 1.7320508f * s));
}

/* 64 x 64 tile, 16 columns of K per step, 4 x 4 results per thread. The sum over K is taken in two
 * levels, so that its rounding error grows with the step length and the number of steps, not with K. */
constexpr int kFgT = 64, kFgK = 16;
__global__ void __launch_bounds__(256)
lm_gemm_f32_kernel(float *y, int ld_out, const float *x, int ldx, const uint16_t *W, int ldw, int M, int N, int K, int act,
                   const int4 *table, int group_rows) {
    __shared__ __align__(16) float xs[kFgK][kFgT + 4], ws[kFgK][kFgT + 4];
    pdl_launch_dependents();
    pdl_wait();
    const int n0 = blockIdx.x * kFgT;
    int m0 = blockIdx.y * kFgT;
    if (table) {                       /* two tiles of rows per block of 128 */
        const int4 g = __ldcg(table + (blockIdx.y >> 1));
        m0 = g.y + (int)(blockIdx.y & 1) * kFgT;
        M = g.y + g.z;
        if (g.x < 0 || m0 >= M) return;
        W += (size_t)g.x * group_rows * ldw;
    }
    const int tid = threadIdx.x, tm = (tid >> 4) * 4, tn = (tid & 15) * 4;
    float sum[4][4] = {};
    for (int k0 = 0; k0 < K; k0 += kFgK) {
        for (int i = tid; i < kFgT * kFgK; i += 256) {
            const int r = i / kFgK, k = i % kFgK;
            const bool kin = k0 + k < K;
            xs[k][r] = kin && m0 + r < M ? x[(size_t)(m0 + r) * ldx + k0 + k] : 0.0f;
            ws[k][r] = kin && n0 + r < N ? __uint_as_float((uint32_t)W[(size_t)(n0 + r) * ldw + k0 + k] << 16) : 0.0f;
        }
        __syncthreads();
        float acc[4][4] = {};
#pragma unroll
        for (int k = 0; k < kFgK; k++) {
            const float4 a = *(const float4 *)&xs[k][tm], b = *(const float4 *)&ws[k][tn];
            const float av[4] = {a.x, a.y, a.z, a.w}, bv[4] = {b.x, b.y, b.z, b.w};
#pragma unroll
            for (int i = 0; i < 4; i++)
#pragma unroll
                for (int j = 0; j < 4; j++) acc[i][j] = fmaf(av[i], bv[j], acc[i][j]);
        }
#pragma unroll
        for (int i = 0; i < 4; i++)
#pragma unroll
            for (int j = 0; j < 4; j++) sum[i][j] += acc[i][j];
        __syncthreads();
    }
    for (int i = 0; i < 4; i++) {
        const int m = m0 + tm + i;
        if (m >= M) break;
        if (act == LM_ACT_SWIGLU) {
            for (int j = 0; j < 4; j += 2) {
                const int n = n0 + tn + j;
                if (n + 1 < N) y[(size_t)m * ld_out + n / 2] = sum[i][j] / (1.0f + expf(-sum[i][j])) * sum[i][j + 1];
            }
        } else {
            for (int j = 0; j < 4; j++) {
                const float v = act == LM_ACT_RELU2 ? fmaxf(sum[i][j], 0.0f) * fmaxf(sum[i][j], 0.0f) : sum[i][j];
                if (n0 + tn + j < N) y[(size_t)m * ld_out + n0 + tn + j] = v;
            }
        }
    }
}

__global__ void __launch_bounds__(1024)
lm_argmax_advance_kernel(LmDyn *dyn, int *tokens, int *log, int log_cap, const LmPart lg, int vocab, int rows) {
    __shared__ float rv[32];
    __shared__ int ri[32];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x;
    float best = -INFINITY;
    int bi = vocab;
    for (int i = tid; i < vocab; i += 1024) {
        const float v = lm_sum(lg, 0, i);
        if (v > best) { best = v; bi = i; }
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) {
        const float ov = __shfl_xor_sync(0xffffffffu, best, o);
        const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
        if (ov > best || (ov == best && oi < bi)) { best = ov; bi = oi; }
    }
    if ((tid & 31) == 0) { rv[tid >> 5] = best; ri[tid >> 5] = bi; }
    __syncthreads();
    if (tid == 0) {
        for (int w = 0; w < 32; w++)
            if (rv[w] > best || (rv[w] == best && ri[w] < bi)) { best = rv[w]; bi = ri[w]; }
        if (bi >= vocab) bi = 0;                /* every logit is NaN */
        tokens[0] = bi;
        if (dyn->logged < log_cap) log[dyn->logged] = bi;
        dyn->logged += 1;
        dyn->pos += rows;
    }
}

inline int ok(cudaError_t e) { return e == cudaSuccess ? 0 : -1; }

} // namespace

int lm_residual(const LmResidual &a, int M, cudaStream_t st) {
    if (M <= 0) return 0;
    const bool v4 = (a.width & 3) == 0;
    const int groups = v4 ? a.width / 4 : a.width;
    const int threads = groups >= 1024 ? 1024 : (groups + 31) / 32 * 32, nv = (groups + threads - 1) / threads;
    const dim3 g(M), b(threads);
    if (v4) {
        if (nv <= 1) return ok(launch_pdl(lm_residual_kernel<4, 1>, g, b, 0, st, a));
        if (nv <= 2) return ok(launch_pdl(lm_residual_kernel<4, 2>, g, b, 0, st, a));
        if (nv <= 4) return ok(launch_pdl(lm_residual_kernel<4, 4>, g, b, 0, st, a));
    } else {
        if (nv <= 1) return ok(launch_pdl(lm_residual_kernel<1, 1>, g, b, 0, st, a));
        if (nv <= 4) return ok(launch_pdl(lm_residual_kernel<1, 4>, g, b, 0, st, a));
        if (nv <= 16) return ok(launch_pdl(lm_residual_kernel<1, 16>, g, b, 0, st, a));
    }
    return -1;
}

int lm_pack_rows(uint16_t *dst, int Kp, int row0, int step, int col0, const uint16_t *src, int rows, int K, cudaStream_t st) {
    const size_t n = (size_t)rows * K;
    if (n == 0) return 0;
    lm_pack_rows_kernel<<<(unsigned)((n + 255) / 256), 256, 0, st>>>(dst, Kp, row0, step, col0, src, rows, K);
    return ok(cudaGetLastError());
}

int lm_widen(float *dst, const uint16_t *src, int n, cudaStream_t st) {
    if (n <= 0) return 0;
    lm_widen_kernel<<<(n + 255) / 256, 256, 0, st>>>(dst, src, n);
    return ok(cudaGetLastError());
}

int lm_fill_random(uint16_t *dst, size_t n, uint32_t seed, float mean, float scale, cudaStream_t st) {
    if (n == 0) return 0;
    lm_fill_random_kernel<<<(unsigned)((n + 255) / 256), 256, 0, st>>>(dst, n, seed, mean, scale);
    return ok(cudaGetLastError());
}

int lm_gemm_f32(float *y, int ld_out, const float *x, int ldx, const uint16_t *W, int ldw, int M, int N, int K, LmAct act,
                cudaStream_t st, const int4 *table, int group_rows) {
    const dim3 g((N + kFgT - 1) / kFgT, (M + kFgT - 1) / kFgT);
    return ok(launch_pdl(lm_gemm_f32_kernel, g, dim3(256), 0, st, y, ld_out, x, ldx, W, ldw, M, N, K, (int)act,
                         table, group_rows));
}

int lm_argmax_advance(LmDyn *dyn, int *tokens, int *log, int log_cap, LmPart logits, int vocab, int rows, cudaStream_t st) {
    return ok(launch_pdl(lm_argmax_advance_kernel, dim3(1), dim3(1024), 0, st, dyn, tokens, log, log_cap, logits, vocab, rows));
}

} // namespace vb
