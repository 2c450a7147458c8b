/*
 * vb_lm_latent.cu - decoder language models: attention over a latent cache. A token leaves one
 * normed latent and one rotated key part, shared by all heads; keys and values are linear in the
 * latent, so that with few rows the key matrix is applied to the query instead (absorb), all heads
 * attend over the same cache rows (attend), and the value matrix is applied to what they read
 * (readout, with the gate per head). Prompts write keys and values out (gather, a GEMM) and use
 * the attention of vb_lm_attn.cu.
 *
 *   lm_latent_prepare  norms of both latents, rotated key part, cache append, gates, angles, routing,
 *                      squared-ReLU columns of a feed-forward that shares the in-projection
 *   lm_latent_attend   mma.sync on hi + lo BF16 halves (cache rows as such halves), or fp32 pipes for
 *                      other sizes and the 32-bit mode; key splits, merged by the readout
 */
#include "vb_lm_attn.cuh"
#include "vb_tc.cuh"

namespace vb {

namespace {

inline int ok(cudaError_t e) { return e == cudaSuccess ? 0 : -1; }

template <typename K> int allow_smem(K *kernel, size_t smem, size_t *set) {
    if (smem <= *set) return 0;
    if (cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
        cudaGetLastError();
        return -1;
    }
    *set = smem;
    return 0;
}

__host__ __device__ constexpr int up4(int v) { return (v + 3) & ~3; }
constexpr size_t kSmemLimit = 216 * 1024;      /* dynamic part; a few KB are static */

/* ------------------------------------------------------------------ a row's latents */
constexpr int kLpThreads = 512, kLpWarps = kLpThreads / 32;      /* at most: as many as a row has float4 columns */

/* The `top` largest of z[0, n), the first one on a tie, and the softmax over them: one warp. `pick` holds `top` indexes. */
VB_DEVINL void route_row(float *z, int n, int top, int *pick, int *chosen, float *weight, int lane) {
    unsigned taken = 0;                      /* bit i: z[lane + 32 * i] */
    float first = 0.0f, sum = 0.0f;
    for (int k = 0; k < top; k++) {
        /* floats as unsigned integers of the same order, so that a warp reduces them in one instruction */
        unsigned best = 0u;
        int bi = 0x7fffffff;
        for (int i = 0, e = lane; e < n; i++, e += 32) {
            const unsigned u = __float_as_uint(z[e]), key = u & 0x80000000u ? ~u : u | 0x80000000u;
            if (!((taken >> i) & 1u) && (bi == 0x7fffffff || key > best)) { best = key; bi = e; }
        }
        const unsigned all = __reduce_max_sync(0xffffffffu, best);
        bi = __reduce_min_sync(0xffffffffu, best == all ? bi : 0x7fffffff);
        if ((bi & 31) == lane) taken |= 1u << (bi >> 5);
        const float v = z[bi];
        if (k == 0) first = v;
        const float p = expf(v - first);
        sum += p;
        __syncwarp();
        if (lane == 0) { pick[k] = bi; z[bi] = p; }      /* this place is not looked at again */
    }
    __syncwarp();
    for (int k = lane; k < top; k += 32) {
        chosen[k] = pick[k];
        weight[k] = z[pick[k]] / sum;
    }
}

/* grid = (rows, 1 + pieces of the feed-forward columns). ONE: the in-projection is not split (many rows), which leaves
 * registers for more CTAs per SM. */
template <bool ONE>
__global__ void __launch_bounds__(kLpThreads, ONE ? 3 : 1) lm_latent_prepare_kernel(const LmLatent a) {
    extern __shared__ __align__(16) float lp[];
    __shared__ float red[2][kLpWarps];
    pdl_launch_dependents();
    pdl_wait();
    const int threads = blockDim.x, warps = threads >> 5;
    const int m = blockIdx.x, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    auto sum4 = [&](int c) { return ONE ? vb_ldcg4(a.in.p + (size_t)m * a.in.ld + c) : lm_sum4(a.in, m, c); };
    auto sum1 = [&](int c) { return ONE ? vb_ldcg(a.in.p + (size_t)m * a.in.ld + c) : lm_sum_batch(a.in, m, c); };
    if (blockIdx.y > 0) {
        const int c = (((int)blockIdx.y - 1) * threads + tid) * 4;
        if (c >= a.ff) return;
        const float4 v = sum4(a.col_ff + c);
        float e[4] = {v.x, v.y, v.z, v.w};
#pragma unroll
        for (int i = 0; i < 4; i++) { e[i] = fmaxf(e[i], 0.0f); e[i] *= e[i]; }
        if (c + 3 < a.ff) {
            lm_put4(a.out, m, a.ff_out + c, e);
        } else {
            for (int i = 0; c + i < a.ff; i++) lm_put(a.out, m, a.ff_out + c + i, e[i]);
        }
        return;
    }
    const int half = a.rot / 2, row = a.rank + a.rot_dim, nq = up4(a.q_rank), nc = a.c_gain ? up4(row) : 0;
    float *ql = lp, *cl = ql + nq, *z = cl + nc, *cs = z + a.experts;
    const int pos = a.dyn->pos + m;
    auto angles = [&]() {
        for (int i = tid; i < half; i += threads) {
            float c, s;
            lm_angle(pos, a.freq[i], a.freq[half + i], a.mag, &c, &s);
            cs[i] = c;
            cs[half + i] = s;
            a.cs[(size_t)m * a.rot + i] = c;
            a.cs[(size_t)m * a.rot + half + i] = s;
        }
    };
    if (!ONE) angles();
    /* a part that does not fill its last four columns is followed by zero ones */
    float sq = 0.0f, sc = 0.0f;
    for (int c = tid * 4; c < nq + nc; c += threads * 4) {
        const bool isq = c < nq;
        const float4 v = sum4(isq ? c : a.col_c + c - nq);
        *reinterpret_cast<float4 *>(lp + c) = v;
        if (isq) {
            sq += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        } else {
            const int d = c - nq;
            sc += (d < a.rank ? v.x * v.x : 0.0f) + (d + 1 < a.rank ? v.y * v.y : 0.0f) + (d + 2 < a.rank ? v.z * v.z : 0.0f) +
                  (d + 3 < a.rank ? v.w * v.w : 0.0f);
        }
    }
    for (int e = tid; e < a.experts; e += threads) z[e] = sum1(a.col_router + e);
    for (int h = tid; h < a.heads; h += threads)
        a.gate[(size_t)m * a.heads + h] = 1.0f / (1.0f + expf(-sum1(a.col_g + h)));
    if (ONE) angles();
    sq = vb_warp_sum(sq);
    sc = vb_warp_sum(sc);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sc; }
    __syncthreads();
    sq = sc = 0.0f;
#pragma unroll
    for (int w = 0; w < kLpWarps; w++)
        if (w < warps) { sq += red[0][w]; sc += red[1][w]; }
    const float rq = 1.0f / sqrtf(sq / (float)a.q_rank + a.eps), rc = 1.0f / sqrtf(sc / (float)a.rank + a.eps);
    if ((a.q_rank & 3) == 0) {
        for (int c = tid * 4; c < a.q_rank; c += threads * 4) {
            const float4 g = __ldg(reinterpret_cast<const float4 *>(a.q_gain + c));
            const float e[4] = {ql[c] * rq * g.x, ql[c + 1] * rq * g.y, ql[c + 2] * rq * g.z, ql[c + 3] * rq * g.w};
            lm_put4(a.q_latent, m, c, e);
        }
    } else {
        for (int c = tid; c < a.q_rank; c += threads) lm_put(a.q_latent, m, c, ql[c] * rq * __ldg(a.q_gain + c));
    }
    if (a.c_gain) {
        float *dst = lm_state(a.kv, a.dyn) + (size_t)lm_ring_row(a.ring, pos) * row;
        auto value = [&](int d) {
            if (d < a.rank) return cl[d] * rc * __ldg(a.c_gain + d);
            const int j = d - a.rank, i = j >> 1;
            if (j >= a.rot) return cl[d];
            return (j & 1) ? cl[d] * cs[i] + cl[d - 1] * cs[half + i] : cl[d] * cs[i] - cl[d + 1] * cs[half + i];
        };
        if ((row & 3) == 0) {
            for (int d = tid * 4; d < row; d += threads * 4)
                kv_put4(dst, row, d, make_float4(value(d), value(d + 1), value(d + 2), value(d + 3)), a.split);
        } else {
            for (int d = tid; d < row; d += threads) kv_put(dst, row, d, value(d), a.split);
        }
    }
    if (a.experts > 0 && warp == warps - 1)
        route_row(z, a.experts, a.top, reinterpret_cast<int *>(cs + a.rot), a.chosen + (size_t)m * a.top, a.weight + (size_t)m * a.top, lane);
}

/* ------------------------------------------------------------------ queries into the latent's space */
constexpr int kLtThreads = 256, kLtWarps = 8;

VB_DEVINL void bf16x8(const uint4 &u, float (&f)[8]) {
    f[0] = vb_bf16_lo(u.x); f[1] = vb_bf16_hi(u.x); f[2] = vb_bf16_lo(u.y); f[3] = vb_bf16_hi(u.y);
    f[4] = vb_bf16_lo(u.z); f[5] = vb_bf16_hi(u.z); f[6] = vb_bf16_lo(u.w); f[7] = vb_bf16_hi(u.w);
}

/* ql[m][h][r] = sum over d of q[m][h][d] * W_key[h * dim + d][r]; the rotated part follows. grid = (heads, 64-column
 * blocks of the latent, MR-row blocks). Eight lanes share a 128-byte piece of a weight row; the weights of the first
 * kPre steps are requested before the previous kernel has ended. */
template <int MR>
__global__ void __launch_bounds__(kLtThreads) lm_latent_absorb_kernel(const LmLatent a, int M) {
    extern __shared__ __align__(16) float ab[];
    __shared__ float red[kLtWarps][MR][64];
    constexpr int kPre = 4;
    const int h = blockIdx.x, kb = blockIdx.y, m0 = blockIdx.z * MR, nr = M - m0 < MR ? M - m0 : MR;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int d0 = warp * 4 + (lane >> 3), c0 = (lane & 7) * 8;
    pdl_launch_dependents();
    uint4 pre[kPre];
#pragma unroll
    for (int i = 0; i < kPre; i++) {
        const int d = d0 + i * 32;
        pre[i] = d < a.dim ? __ldg(reinterpret_cast<const uint4 *>(lm_weight_row(a.ukv, h * a.dim + d, kb) + c0)) : make_uint4(0u, 0u, 0u, 0u);
    }
    pdl_wait();
    const int hw = a.dim + a.rot_dim, row = a.rank + a.rot_dim;
    for (int i = tid; i < MR * a.dim; i += kLtThreads) {
        const int r = i / a.dim, d = i % a.dim;
        ab[i] = r < nr ? lm_sum_batch(a.q, m0 + r, h * hw + d) : 0.0f;
    }
    if (kb == 0) {
        const int half = a.rot / 2;
        for (int i = tid; i < nr * a.rot_dim; i += kLtThreads) {
            const int r = i / a.rot_dim, j = i % a.rot_dim, m = m0 + r, k = j >> 1;
            float v = lm_sum_batch(a.q, m, h * hw + a.dim + j);
            if (j < a.rot) {
                const float u = lm_sum_batch(a.q, m, h * hw + a.dim + (j ^ 1));
                const float c = a.cs[(size_t)m * a.rot + k], s = a.cs[(size_t)m * a.rot + half + k];
                v = (j & 1) ? v * c + u * s : v * c - u * s;
            }
            a.ql[((size_t)m * a.heads + h) * row + a.rank + j] = v;
        }
    }
    __syncthreads();
    float acc[MR][8];
#pragma unroll
    for (int r = 0; r < MR; r++)
#pragma unroll
        for (int j = 0; j < 8; j++) acc[r][j] = 0.0f;
    auto add = [&](const uint4 &u, int d) {
        float w[8];
        bf16x8(u, w);
#pragma unroll
        for (int r = 0; r < MR; r++) {
            const float q = ab[r * a.dim + d];
#pragma unroll
            for (int j = 0; j < 8; j++) acc[r][j] = fmaf(q, w[j], acc[r][j]);
        }
    };
#pragma unroll
    for (int i = 0; i < kPre; i++)
        if (d0 + i * 32 < a.dim) add(pre[i], d0 + i * 32);
    for (int d = d0 + kPre * 32; d < a.dim; d += 32)
        add(__ldg(reinterpret_cast<const uint4 *>(lm_weight_row(a.ukv, h * a.dim + d, kb) + c0)), d);
#pragma unroll
    for (int r = 0; r < MR; r++)
#pragma unroll
        for (int j = 0; j < 8; j++) {
            float v = acc[r][j];
            v += __shfl_xor_sync(0xffffffffu, v, 8);
            v += __shfl_xor_sync(0xffffffffu, v, 16);
            if (lane < 8) red[warp][r][c0 + j] = v;
        }
    __syncthreads();
    for (int i = tid; i < nr * 64; i += kLtThreads) {
        const int r = i >> 6, c = i & 63, col = kb * 64 + c;
        if (col >= a.rank) continue;
        float v = 0.0f;
#pragma unroll
        for (int w = 0; w < kLtWarps; w++) v += red[w][r][c];
        a.ql[((size_t)(m0 + r) * a.heads + h) * row + col] = v;
    }
}

/* ------------------------------------------------------------------ attention over cache rows */
constexpr int kLaPairs = kLmLatentPairs, kLaSplits = 64, kLaBudget = 148;

inline int attend_tiles(int M, int heads) { return (M * heads + kLaPairs - 1) / kLaPairs; }
inline int attend_splits(int M, int heads) {
    const int s = kLaBudget / attend_tiles(M, heads);
    return s < 1 ? 1 : s > kLaSplits ? kLaSplits : s;
}

/* Key tiles of pairs p0 .. p0 + np - 1 (pair = row * heads + head). */
template <int KT>
VB_DEVINL KeyTiles pair_tiles(const LmLatent &a, int M, int p0, int *np) {
    const int P = M * a.heads, pos0 = a.dyn->pos;
    *np = P - p0 < kLaPairs ? P - p0 : kLaPairs;
    return key_tiles<KT>(pos0 + p0 / a.heads, pos0 + (p0 + *np - 1) / a.heads, a.window, 0);
}

/* What a key split leaves: [split][pair][rank] sums of weighted rows, then [split][pair] (largest score, sum of weights). */
VB_DEVINL float2 *attend_stats(const LmLatent &a, int splits, int P) {
    return reinterpret_cast<float2 *>(a.scratch + (((size_t)splits * P * a.rank + 1) & ~(size_t)1));
}

constexpr int kLaKeys = 32;

constexpr int kLaThreads = 512, kLaWarps = 16;
static_assert(kLaWarps == kLaPairs, "a warp owns the softmax of one pair");

struct AttendSmem {
    int row_bytes;               /* of a query or key row in one plane: whole 64-element groups */
    size_t q, k, total;
    int stages;
};
inline AttendSmem attend_smem(int rank, int rot_dim) {
    AttendSmem s;
    s.row_bytes = (rank + rot_dim + 63) / 64 * 128;
    s.q = (size_t)2 * kLaPairs * s.row_bytes;
    s.k = (size_t)2 * kLaKeys * s.row_bytes;
    s.stages = s.q + 2 * s.k <= kSmemLimit ? 2 : 1;
    s.total = s.q + s.stages * s.k;
    return s;
}

/* A CTA attends with 16 (row, head) pairs over its share of the visible cache rows, 32 at a time. Scores: a warp takes
 * eight keys and a quarter of the columns; values: a warp takes every 16th 16-column step. Products a.b as
 * a_hi.b_hi + a_hi.b_lo + a_lo.b_hi, accumulated in fp32. ND: value steps per warp. grid = (pair tiles, splits) */
template <int ND>
__global__ void __launch_bounds__(kLaThreads) lm_latent_attend_kernel(const LmLatent a, int M, int row_bytes, int stages) {
    extern __shared__ __align__(128) unsigned char at_smem[];
    __shared__ float S[4][kLaPairs][kLaKeys + 1], mx[kLaPairs], den[kLaPairs], cor[kLaPairs];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int q_plane = kLaPairs * row_bytes, k_plane = kLaKeys * row_bytes;
    unsigned char *Kb = at_smem + 2 * q_plane;
    pdl_launch_dependents();
    const int row = a.rank + a.rot_dim, per = row / 8, chunks = row_bytes / 16;
    auto swz = [&](int r, int chunk) { return (uint32_t)(r * row_bytes + (((chunk & ~7) | ((chunk ^ r) & 7)) << 4)); };
    /* what is never loaded: columns beyond the row, in every plane */
    for (int r = warp; per < chunks && r < 2 * kLaPairs + stages * 2 * kLaKeys; r += kLaWarps) {
        const bool isq = r < 2 * kLaPairs;
        const int k = r - 2 * kLaPairs;
        unsigned char *plane = isq ? at_smem + (r / kLaPairs) * q_plane : Kb + (k / kLaKeys) * k_plane;
        const int rr = isq ? r % kLaPairs : k % kLaKeys;
        for (int c = per + lane; c < chunks; c += 32) *reinterpret_cast<uint4 *>(plane + swz(rr, c)) = make_uint4(0u, 0u, 0u, 0u);
    }
    pdl_wait();
    int np;
    const int p0 = blockIdx.x * kLaPairs, sp = blockIdx.y;
    const KeyTiles kt = pair_tiles<kLaKeys>(a, M, p0, &np);
    const int S_eff = (int)gridDim.y < kt.n_tiles ? (int)gridDim.y : kt.n_tiles;
    if (sp >= S_eff) return;
    const int t0 = (int)((long long)kt.n_tiles * sp / S_eff), t1 = (int)((long long)kt.n_tiles * (sp + 1) / S_eff);
    const int pos0 = a.dyn->pos, P = M * a.heads;
    const float *cache = lm_state(a.kv, a.dyn);
    auto request = [&](int t) {
        int j0, n;
        key_tile<kLaKeys>(kt, t, &j0, &n);
        unsigned char *b = Kb + (stages == 2 ? (t & 1) : 0) * 2 * k_plane;
        for (int key = warp; key < n; key += kLaWarps) {
            const uint16_t *src = reinterpret_cast<const uint16_t *>(cache + (size_t)lm_ring_row(a.ring, j0 + key) * row);
            for (int f = lane; f < 2 * per; f += 32) {
                const int plane = f >= per ? 1 : 0;
                lm_cp16(b + plane * k_plane + swz(key, f - plane * per), src + f * 8);
            }
        }
        /* beyond the last key: weights of zero must not meet what an earlier launch left */
        for (int key = n + warp; key < kLaKeys; key += kLaWarps)
            for (int f = lane; f < 2 * per; f += 32) {
                const int plane = f >= per ? 1 : 0;
                *reinterpret_cast<uint4 *>(b + plane * k_plane + swz(key, f - plane * per)) = make_uint4(0u, 0u, 0u, 0u);
            }
        lm_cp_commit();
    };
    request(t0);
    for (int p = warp; p < kLaPairs; p += kLaWarps) {
        const float *q = a.ql + (size_t)(p0 + p) * row;
        for (int chunk = lane; chunk < per; chunk += 32) {
            uint32_t hi[8] = {}, lo[8] = {};
            if (p < np) {
                const float4 u = vb_ldcg4(q + chunk * 8), v = vb_ldcg4(q + chunk * 8 + 4);
                const float e[8] = {u.x, u.y, u.z, u.w, v.x, v.y, v.z, v.w};
#pragma unroll
                for (int j = 0; j < 8; j++) hilo(e[j], hi[j], lo[j]);
            }
            unsigned char *o = at_smem + swz(p, chunk);
            *reinterpret_cast<uint4 *>(o) = make_uint4(hi[0] | (hi[1] << 16), hi[2] | (hi[3] << 16), hi[4] | (hi[5] << 16), hi[6] | (hi[7] << 16));
            *reinterpret_cast<uint4 *>(o + q_plane) =
                make_uint4(lo[0] | (lo[1] << 16), lo[2] | (lo[3] << 16), lo[4] | (lo[5] << 16), lo[6] | (lo[7] << 16));
        }
    }
    if (tid < kLaPairs) { mx[tid] = -INFINITY; den[tid] = 0.0f; }
    float o[2 * ND][4];
#pragma unroll
    for (int i = 0; i < 2 * ND; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    const int steps = row_bytes / 32, vsteps = (a.rank + 15) / 16;
    const int nt = warp & 3, kh = warp >> 2, mat = lane >> 3, mr = lane & 7;
    const uint32_t sQ = vb_smem_u32(at_smem);

    for (int t = t0; t < t1; t++) {
        int j0, n;
        key_tile<kLaKeys>(kt, t, &j0, &n);
        if (stages == 1 && t > t0) {
            __syncthreads();
            request(t);
        }
        lm_cp_wait_all();
        __syncthreads();
        if (stages == 2 && t + 1 < t1) request(t + 1);
        const uint32_t sK = vb_smem_u32(Kb + (stages == 2 ? (t & 1) : 0) * 2 * k_plane);
        float s0[4] = {}, s1[4] = {}, s2[4] = {};
#pragma unroll 4
        for (int ks = kh * (steps / 4); ks < (kh + 1) * (steps / 4); ks++) {      /* rows are whole 64-element groups */
            uint32_t qh[4], ql[4], b[4];
            const uint32_t qo = swz((lane & 7) + ((lane >> 3) & 1) * 8, ks * 2 + (lane >> 4));
            ldsm(qh, sQ + qo);
            ldsm(ql, sQ + q_plane + qo);
            ldsm(b, sK + (mat >> 1) * k_plane + swz(nt * 8 + mr, ks * 2 + (mat & 1)));     /* high halves, low halves */
            mma_bf16(s0, qh, b[0], b[1]);
            mma_bf16(s1, qh, b[2], b[3]);
            mma_bf16(s2, ql, b[0], b[1]);
        }
#pragma unroll
        for (int c = 0; c < 4; c++) S[kh][gq + (c >> 1) * 8][nt * 8 + 2 * tq + (c & 1)] = s0[c] + (s1[c] + s2[c]);
        __syncthreads();
        {
            const int p = warp, pc = p0 + p < P ? p0 + p : P - 1;
            const int i = pos0 + pc / a.heads;
            float s = ((S[0][p][lane] + S[1][p][lane]) + (S[2][p][lane] + S[3][p][lane])) * a.scale;
            if (lane >= n || !key_seen(i, j0 + lane, a.window, 0)) s = -INFINITY;
            float top = s;
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, off));
            const float old = mx[p], now = fmaxf(old, top), ref = now > -INFINITY ? now : 0.0f;
            const float w = expf(s - ref);
            const float sum = vb_warp_sum(w);
            S[0][p][lane] = w;
            __syncwarp();
            if (lane == 0) {
                const float c = expf(old - ref);
                cor[p] = c;
                mx[p] = now;
                den[p] = den[p] * c + sum;
            }
        }
        __syncthreads();
        uint32_t ph[2][4], pl[2][4];
#pragma unroll
        for (int kp = 0; kp < 2; kp++)
#pragma unroll
            for (int x = 0; x < 4; x++) {
                const float *w = &S[0][gq + (x & 1) * 8][kp * 16 + (x >> 1) * 8 + 2 * tq];
                uint32_t h0, l0, h1, l1;
                hilo(w[0], h0, l0);
                hilo(w[1], h1, l1);
                ph[kp][x] = h0 | (h1 << 16);
                pl[kp][x] = l0 | (l1 << 16);
            }
        const float cA = cor[gq], cB = cor[gq + 8];
#pragma unroll
        for (int i = 0; i < ND; i++) {
            const int dp = warp + i * kLaWarps;
            if (dp >= vsteps) break;
#pragma unroll
            for (int u = 0; u < 2; u++) { o[2 * i + u][0] *= cA; o[2 * i + u][1] *= cA; o[2 * i + u][2] *= cB; o[2 * i + u][3] *= cB; }
#pragma unroll
            for (int kp = 0; kp < 2; kp++) {
                const uint32_t off = swz(kp * 16 + (mat & 1) * 8 + mr, dp * 2 + (mat >> 1));
                uint32_t vh[4], vl[4];
                ldsm_t(vh, sK + off);
                ldsm_t(vl, sK + k_plane + off);
                mma_bf16(o[2 * i], ph[kp], vh[0], vh[1]);
                mma_bf16(o[2 * i + 1], ph[kp], vh[2], vh[3]);
                mma_bf16(o[2 * i], ph[kp], vl[0], vl[1]);
                mma_bf16(o[2 * i + 1], ph[kp], vl[2], vl[3]);
                mma_bf16(o[2 * i], pl[kp], vh[0], vh[1]);
                mma_bf16(o[2 * i + 1], pl[kp], vh[2], vh[3]);
            }
        }
    }
    /* (the last statistics were written before the barrier ahead of the value products) */
    float *out = a.scratch + ((size_t)sp * P + p0) * a.rank;
#pragma unroll
    for (int i = 0; i < ND; i++) {
        const int dp = warp + i * kLaWarps;
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int c = dp * 16 + u * 8 + 2 * tq;
            if (c >= a.rank) continue;
            if (gq < np) *reinterpret_cast<float2 *>(out + (size_t)gq * a.rank + c) = make_float2(o[2 * i + u][0], o[2 * i + u][1]);
            if (gq + 8 < np) *reinterpret_cast<float2 *>(out + (size_t)(gq + 8) * a.rank + c) = make_float2(o[2 * i + u][2], o[2 * i + u][3]);
        }
    }
    if (tid < np) attend_stats(a, (int)gridDim.y, P)[(size_t)sp * P + p0 + tid] = make_float2(mx[tid], den[tid]);
}

/* The same on the fp32 pipes, any sizes; cache rows in either form. */
inline size_t attend_f32_smem(int rank, int rot_dim, int keys) {
    const size_t row = (size_t)rank + rot_dim;
    return sizeof(float) * (kLaPairs * row + keys * (row + 1) + kLaPairs * (size_t)rank + kLaPairs * (keys + 1) + 3 * kLaPairs);
}
inline int attend_f32_keys(int rank, int rot_dim) { return attend_f32_smem(rank, rot_dim, 32) <= kSmemLimit ? 32 : 8; }

template <int KT>
__global__ void __launch_bounds__(kLtThreads) lm_latent_attend_f32_kernel(const LmLatent a, int M) {
    extern __shared__ __align__(16) float af[];
    pdl_launch_dependents();
    pdl_wait();
    int np;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int p0 = blockIdx.x * kLaPairs, sp = blockIdx.y, row = a.rank + a.rot_dim, pos0 = a.dyn->pos, P = M * a.heads;
    const KeyTiles kt = pair_tiles<KT>(a, M, p0, &np);
    const int S_eff = (int)gridDim.y < kt.n_tiles ? (int)gridDim.y : kt.n_tiles;
    if (sp >= S_eff) return;
    const int t0 = (int)((long long)kt.n_tiles * sp / S_eff), t1 = (int)((long long)kt.n_tiles * (sp + 1) / S_eff);
    float *Q = af, *K = Q + kLaPairs * row, *O = K + KT * (row + 1), *S = O + kLaPairs * a.rank, *mx = S + kLaPairs * (KT + 1),
          *den = mx + kLaPairs, *cor = den + kLaPairs;
    const float *cache = lm_state(a.kv, a.dyn);
    for (int i = tid; i < np * row; i += kLtThreads) Q[i] = __ldcg(a.ql + (size_t)p0 * row + i);
    for (int i = tid; i < np * a.rank; i += kLtThreads) O[i] = 0.0f;
    if (tid < kLaPairs) { mx[tid] = -INFINITY; den[tid] = 0.0f; }
    for (int t = t0; t < t1; t++) {
        int j0, n;
        key_tile<KT>(kt, t, &j0, &n);
        __syncthreads();
        for (int i = tid; i < n * row; i += kLtThreads) {
            const int j = i / row, d = i % row;
            K[j * (row + 1) + d] = kv_get(cache + (size_t)lm_ring_row(a.ring, j0 + j) * row, row, d, a.split);
        }
        __syncthreads();
        for (int p = warp; p < np; p += kLtWarps) {
            const int i = pos0 + (p0 + p) / a.heads;
            float s = -INFINITY;
            if (lane < n && key_seen(i, j0 + lane, a.window, 0)) {
                const float *q = Q + p * row, *k = K + lane * (row + 1);
                float e0 = 0.0f, e1 = 0.0f, e2 = 0.0f, e3 = 0.0f;
                int d = 0;
                for (; d + 3 < row; d += 4) {
                    e0 = fmaf(q[d], k[d], e0);
                    e1 = fmaf(q[d + 1], k[d + 1], e1);
                    e2 = fmaf(q[d + 2], k[d + 2], e2);
                    e3 = fmaf(q[d + 3], k[d + 3], e3);
                }
                for (; d < row; d++) e0 = fmaf(q[d], k[d], e0);
                s = ((e0 + e1) + (e2 + e3)) * a.scale;
            }
            float top = s;
#pragma unroll
            for (int off = 16; off > 0; off >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, off));
            const float old = mx[p], now = fmaxf(old, top), ref = now > -INFINITY ? now : 0.0f;
            const float w = expf(s - ref);
            const float sum = vb_warp_sum(w);
            if (lane < KT) S[p * (KT + 1) + lane] = w;
            __syncwarp();
            if (lane == 0) {
                const float c = expf(old - ref);
                cor[p] = c;
                mx[p] = now;
                den[p] = den[p] * c + sum;
            }
        }
        __syncthreads();
        for (int i = tid; i < np * a.rank; i += kLtThreads) {
            const int p = i / a.rank, d = i % a.rank;
            float o = O[i] * cor[p];
            for (int j = 0; j < n; j++) o = fmaf(S[p * (KT + 1) + j], K[j * (row + 1) + d], o);
            O[i] = o;
        }
    }
    __syncthreads();
    float *out = a.scratch + ((size_t)sp * P + p0) * a.rank;
    for (int i = tid; i < np * a.rank; i += kLtThreads) out[i] = O[i];
    if (tid < np) attend_stats(a, (int)gridDim.y, P)[(size_t)sp * P + p0 + tid] = make_float2(mx[tid], den[tid]);
}

/* ------------------------------------------------------------------ values */
/* Merges the key splits of a head (in order), applies its value matrix and its gate. grid = (heads, 32-row blocks of the
 * value matrix, MR-row blocks). KT: keys per tile of the kernel that wrote the splits. */
template <int MR, int KT>
__global__ void __launch_bounds__(kLtThreads) lm_latent_readout_kernel(const LmLatent a, int M, int splits) {
    extern __shared__ __align__(16) float ro[];                /* [MR][rank, padded to 64] */
    __shared__ float wgt[MR][kLaSplits];
    __shared__ int count[MR];
    constexpr int kPre = MR == 1 ? 8 : 1;
    const int h = blockIdx.x, m0 = blockIdx.z * MR, nr = M - m0 < MR ? M - m0 : MR;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int v = blockIdx.y * 32 + warp * 4 + (lane >> 3), c0 = (lane & 7) * 8;
    const int kblocks = (a.rank + 63) / 64, rp = kblocks * 64;
    const int wrow = a.heads * a.dim + h * a.vdim + (v < a.vdim ? v : 0);
    pdl_launch_dependents();
    uint4 pre[kPre];
#pragma unroll
    for (int i = 0; i < kPre; i++)
        pre[i] = i < kblocks ? __ldg(reinterpret_cast<const uint4 *>(lm_weight_row(a.ukv, wrow, i) + c0)) : make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    const size_t P = (size_t)M * a.heads;
    const float2 *stats = attend_stats(a, splits, (int)P);
    if (warp < nr) {
        const int p = (m0 + warp) * a.heads + h;
        int np;
        const KeyTiles kt = pair_tiles<KT>(a, M, p / kLaPairs * kLaPairs, &np);
        const int S = splits < kt.n_tiles ? splits : kt.n_tiles;
        float2 st[2];
        float mu[2], top = -INFINITY, L = 0.0f;
#pragma unroll
        for (int x = 0; x < 2; x++) {
            const int u = lane + 32 * x;
            st[x] = u < S ? __ldcg(stats + u * P + p) : make_float2(-INFINITY, 0.0f);
            top = fmaxf(top, st[x].x);
        }
#pragma unroll
        for (int off = 16; off > 0; off >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, off));
#pragma unroll
        for (int x = 0; x < 2; x++) {
            mu[x] = expf(st[x].x - top);                       /* a row always sees itself: top is finite */
            L = fmaf(mu[x], st[x].y, L);
        }
        L = vb_warp_sum(L);
        wgt[warp][lane] = mu[0] / L;
        wgt[warp][lane + 32] = mu[1] / L;
        if (lane == 0) count[warp] = S;
    }
    __syncthreads();
    if ((a.rank & 3) == 0) {
        /* four columns per item; where there are few items, neighbouring lanes share one and take every second,
         * fourth, ... split */
        const int nv = a.rank / 4, items = nr * nv;
        int parts = 1;
        while (parts < 8 && items * parts * 2 <= kLtThreads) parts *= 2;
        for (int i0 = 0; i0 < items; i0 += kLtThreads / parts) {
            const int i = i0 + tid / parts, part = tid % parts;
            const bool in = i < items;
            const int r = in ? i / nv : 0, c = in ? i % nv * 4 : 0;
            const float *s = a.scratch + ((size_t)(m0 + r) * a.heads + h) * a.rank + c;
            const int S = in ? count[r] : 0;
            float4 o = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
            for (int u = part; u < S; u += parts) {
                const float4 t = vb_ldcg4(s + u * P * a.rank);
                const float w = wgt[r][u];
                o.x = fmaf(w, t.x, o.x); o.y = fmaf(w, t.y, o.y); o.z = fmaf(w, t.z, o.z); o.w = fmaf(w, t.w, o.w);
            }
            for (int off = 1; off < parts; off <<= 1) {
                o.x += __shfl_xor_sync(0xffffffffu, o.x, off); o.y += __shfl_xor_sync(0xffffffffu, o.y, off);
                o.z += __shfl_xor_sync(0xffffffffu, o.z, off); o.w += __shfl_xor_sync(0xffffffffu, o.w, off);
            }
            if (in && part == 0) *reinterpret_cast<float4 *>(ro + r * rp + c) = o;
        }
    } else {
        for (int i = tid; i < nr * a.rank; i += kLtThreads) {
            const int r = i / a.rank, c = i % a.rank, S = count[r];
            const float *s = a.scratch + ((size_t)(m0 + r) * a.heads + h) * a.rank + c;
            float o = 0.0f;
            for (int u = 0; u < S; u++) o = fmaf(wgt[r][u], __ldcg(s + u * P * a.rank), o);
            ro[r * rp + c] = o;
        }
    }
    for (int i = tid; i < nr * (rp - a.rank); i += kLtThreads) ro[i / (rp - a.rank) * rp + a.rank + i % (rp - a.rank)] = 0.0f;
    __syncthreads();
    float acc[MR];
#pragma unroll
    for (int r = 0; r < MR; r++) acc[r] = 0.0f;
    auto add = [&](const uint4 &u, int kb) {
        float w[8];
        bf16x8(u, w);
#pragma unroll
        for (int r = 0; r < MR; r++) {
            if (r >= nr) break;
            const float *x = ro + r * rp + kb * 64 + c0;
#pragma unroll
            for (int j = 0; j < 8; j++) acc[r] = fmaf(w[j], x[j], acc[r]);
        }
    };
#pragma unroll
    for (int i = 0; i < kPre; i++)
        if (i < kblocks) add(pre[i], i);
    for (int kb = kPre; kb < kblocks; kb++) add(__ldg(reinterpret_cast<const uint4 *>(lm_weight_row(a.ukv, wrow, kb) + c0)), kb);
#pragma unroll
    for (int r = 0; r < MR; r++) {
#pragma unroll
        for (int off = 4; off > 0; off >>= 1) acc[r] += __shfl_xor_sync(0xffffffffu, acc[r], off);
        if (r < nr && (lane & 7) == 0 && v < a.vdim)
            lm_put(a.out, m0 + r, h * a.vdim + v, acc[r] * a.gate[(size_t)(m0 + r) * a.heads + h]);
    }
}

/* ------------------------------------------------------------------ latents of a stretch as GEMM rows */
__global__ void lm_latent_gather_kernel(const LmLatent a, uint16_t *terms, int rows_pad, int ld, int first, int n) {
    pdl_launch_dependents();
    pdl_wait();
    const int per = a.rank / 8, row = a.rank + a.rot_dim;
    const size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= (size_t)n * 2 * per) return;
    const int j = (int)(i / (2 * per)), f = (int)(i % (2 * per)), plane = f >= per ? 1 : 0, chunk = f - plane * per;
    const uint16_t *src = reinterpret_cast<const uint16_t *>(lm_state(a.kv, a.dyn) + (size_t)lm_ring_row(a.ring, first + j) * row) +
                          (size_t)plane * row + chunk * 8;
    *reinterpret_cast<uint4 *>(terms + ((size_t)plane * rows_pad + j) * ld + chunk * 8) = __ldcg(reinterpret_cast<const uint4 *>(src));
}

template <bool ONE>
int launch_prepare(const LmLatent &a, int M, cudaStream_t st) {
    static size_t set = 40 * 1024;
    const int columns = up4(a.q_rank) + (a.c_gain ? up4(a.rank + a.rot_dim) : 0);
    const size_t smem = sizeof(float) * ((size_t)columns + a.experts + a.rot + a.top);
    if (allow_smem(lm_latent_prepare_kernel<ONE>, smem, &set)) return -1;
    const int threads = columns >= kLpThreads * 4 ? kLpThreads : columns <= 512 ? 128 : (columns / 4 + 31) / 32 * 32;
    const int pieces = (a.ff + threads * 4 - 1) / (threads * 4);
    return ok(launch_pdl(lm_latent_prepare_kernel<ONE>, dim3(M, 1 + pieces), dim3(threads), smem, st, a));
}

template <int ND>
int launch_attend(const LmLatent &a, int M, const AttendSmem &s, cudaStream_t st) {
    static size_t set = 32 * 1024;
    if (allow_smem(lm_latent_attend_kernel<ND>, s.total, &set)) return -1;
    return ok(launch_pdl(lm_latent_attend_kernel<ND>, dim3(attend_tiles(M, a.heads), attend_splits(M, a.heads)), dim3(kLaThreads), s.total, st, a, M,
                         s.row_bytes, s.stages));
}
template <int KT>
int launch_attend_f32(const LmLatent &a, int M, cudaStream_t st) {
    static size_t set = 32 * 1024;
    const size_t smem = attend_f32_smem(a.rank, a.rot_dim, KT);
    if (allow_smem(lm_latent_attend_f32_kernel<KT>, smem, &set)) return -1;
    return ok(launch_pdl(lm_latent_attend_f32_kernel<KT>, dim3(attend_tiles(M, a.heads), attend_splits(M, a.heads)), dim3(kLtThreads), smem, st, a, M));
}
template <int MR, int KT>
int launch_readout(const LmLatent &a, int M, cudaStream_t st) {
    static size_t set = 32 * 1024;
    const size_t smem = sizeof(float) * MR * ((a.rank + 63) / 64 * 64);
    if (allow_smem(lm_latent_readout_kernel<MR, KT>, smem, &set)) return -1;
    return ok(launch_pdl(lm_latent_readout_kernel<MR, KT>, dim3(a.heads, (a.vdim + 31) / 32, (M + MR - 1) / MR), dim3(kLtThreads), smem, st, a, M,
                         attend_splits(M, a.heads)));
}
template <int MR>
int launch_absorb(const LmLatent &a, int M, cudaStream_t st) {
    static size_t set = 24 * 1024;
    const size_t smem = sizeof(float) * MR * a.dim;
    if (allow_smem(lm_latent_absorb_kernel<MR>, smem, &set)) return -1;
    return ok(launch_pdl(lm_latent_absorb_kernel<MR>, dim3(a.heads, (a.rank + 63) / 64, (M + MR - 1) / MR), dim3(kLtThreads), smem, st, a, M));
}

} // namespace

bool lm_latent_split_ok(int rank, int rot_dim) {
    return rank % 8 == 0 && rot_dim % 8 == 0 && rank <= 1024 && attend_smem(rank, rot_dim).total <= kSmemLimit;
}
bool lm_latent_supported(int q_rank, int rank, int rot_dim) {
    return attend_f32_smem(rank, rot_dim, attend_f32_keys(rank, rot_dim)) <= kSmemLimit &&
           sizeof(float) * ((size_t)q_rank + rank + 2 * rot_dim + 2 * kLmMoeExperts + 16) <= kSmemLimit;
}
size_t lm_latent_scratch_floats(int rows, int heads, int rank) {
    size_t n = 0;
    for (int M = 1; M <= rows; M++) n = n > (size_t)attend_splits(M, heads) * M ? n : (size_t)attend_splits(M, heads) * M;
    return n * heads * (rank + 2) + 2;
}

int lm_latent_prepare(const LmLatent &a, int M, cudaStream_t st) {
    return a.in.n == 1 && M > 64 ? launch_prepare<true>(a, M, st) : launch_prepare<false>(a, M, st);
}

int lm_latent_absorb(const LmLatent &a, int M, cudaStream_t st) { return M == 1 ? launch_absorb<1>(a, M, st) : launch_absorb<8>(a, M, st); }

int lm_latent_attend(const LmLatent &a, int M, cudaStream_t st) {
    if (a.split) {
        const AttendSmem s = attend_smem(a.rank, a.rot_dim);
        if (a.rank <= 256) return launch_attend<1>(a, M, s, st);
        return a.rank <= 512 ? launch_attend<2>(a, M, s, st) : launch_attend<4>(a, M, s, st);
    }
    return attend_f32_keys(a.rank, a.rot_dim) == 32 ? launch_attend_f32<32>(a, M, st) : launch_attend_f32<8>(a, M, st);
}

int lm_latent_readout(const LmLatent &a, int M, cudaStream_t st) {
    if (a.split || attend_f32_keys(a.rank, a.rot_dim) == 32) return M == 1 ? launch_readout<1, 32>(a, M, st) : launch_readout<8, 32>(a, M, st);
    return M == 1 ? launch_readout<1, 8>(a, M, st) : launch_readout<8, 8>(a, M, st);
}

int lm_latent_gather(const LmLatent &a, uint16_t *terms, int rows_pad, int ld, int first, int n, cudaStream_t st) {
    const size_t items = (size_t)n * 2 * (a.rank / 8);
    return ok(launch_pdl(lm_latent_gather_kernel, dim3((unsigned)((items + 255) / 256)), dim3(256), 0, st, a, terms, rows_pad, ld, first, n));
}

} // namespace vb
