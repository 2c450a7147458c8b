/*
 * vb_lm_attn.cu - decoder language models: softmax attention over a ring cache. Query and key
 * norm over the whole projection, rotary positions on a part of the head, optional softcap,
 * optional sliding window with kept first tokens; any head sizes, separate key and value sizes.
 *
 *   lm_attn_prepare  one row per CTA: sums the projection's split-K partials, norms and rotates q
 *                    and k, appends k and v to the cache
 *   lm_attn_generic  fp32 pipes: any sizes, short portions and the 32-bit mode (keys split over CTAs,
 *                    last arrival merges)
 *   lm_attn_step     one token, preparation included
 *   lm_attn_mma      prompts: mma.sync on hi + lo BF16 halves of q, k, v and the weights; the cache keeps
 *                    k and v as such halves
 *
 * Keys are visited in two stretches, the kept first tokens and the window; a stretch that is out
 * of reach of all of a CTA's rows is never loaded.
 */
#include "vb_lm_attn.cuh"
#include "vb_tc.cuh"

namespace vb {

namespace {

inline int ok(cudaError_t e) { return e == cudaSuccess ? 0 : -1; }

/* ------------------------------------------------------------------ q, k, v of a row */
constexpr int kPrepThreads = 512;

__global__ void __launch_bounds__(kPrepThreads) lm_attn_prepare_kernel(const LmAttn a) {
    extern __shared__ __align__(16) float prep_smem[];
    __shared__ float red[2][kPrepThreads / 32];
    const int nq = a.heads * a.dim, nk = a.kv_heads * a.dim, nv = a.kv_heads * a.vdim;
    float *buf = prep_smem;                       /* [nq + nk] */
    float *cs = buf + nq + nk;                    /* [rot / 2] cos, then [rot / 2] sin */
    pdl_launch_dependents();
    pdl_wait();
    const int m = blockIdx.x, tid = threadIdx.x, half = a.rot / 2;
    const int pos = a.dyn->pos + m;
    const size_t row = (size_t)lm_ring_row(a.ring, pos);
    for (int i = tid; i < half; i += kPrepThreads) {
        lm_angle(pos, a.freq[i], a.freq[half + i], a.mag, &cs[i], &cs[half + i]);
    }
    float sq = 0.0f, sk = 0.0f;
    float *Vr = lm_state(a.v, a.dyn) + row * nv;
    if (((nq | nk | a.vdim) & 3) == 0) {
        for (int c = tid * 4; c < nq + nk + nv; c += kPrepThreads * 4) {
            const float4 v = lm_sum4(a.qkv, m, c);
            if (c < nq + nk) {
                const float ss = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
                *reinterpret_cast<float4 *>(buf + c) = v;
                if (c < nq) sq += ss; else sk += ss;
            } else {
                const int j = c - nq - nk, d = j % a.vdim;
                kv_put4(Vr + j - d, a.vdim, d, v, a.split);
            }
        }
    } else {
        for (int c = tid; c < nq + nk; c += kPrepThreads) {
            const float v = lm_sum_batch(a.qkv, m, c);
            buf[c] = v;
            if (c < nq) sq += v * v; else sk += v * v;
        }
        for (int c = tid; c < nv; c += kPrepThreads)
            kv_put(Vr + c / a.vdim * a.vdim, a.vdim, c % a.vdim, lm_sum_batch(a.qkv, m, nq + nk + c), a.split);
    }
    sq = vb_warp_sum(sq);
    sk = vb_warp_sum(sk);
    if ((tid & 31) == 0) { red[0][tid >> 5] = sq; red[1][tid >> 5] = sk; }
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < kPrepThreads / 32; w++) { sq += red[0][w]; sk += red[1][w]; }
    const float rq = 1.0f / sqrtf(sq / (float)nq + a.eps), rk = 1.0f / sqrtf(sk / (float)nk + a.eps);
    float *Kr = lm_state(a.k, a.dyn) + row * nk, *Q = a.q + (size_t)m * nq;
    auto value = [&](int c) {                     /* column c normed and rotated */
        const bool isq = c < nq;
        const int j = isq ? c : c - nq, d = j % a.dim;
        const float *gain = isq ? a.q_gain : a.k_gain;
        const float r = isq ? rq : rk;
        float v = buf[c] * r * __ldg(gain + j);
        if (d < a.rot) {
            const int i = d < half ? d : d - half, other = d < half ? half : -half;
            const float u = buf[c + other] * r * __ldg(gain + j + other);
            v = d < half ? v * cs[i] - u * cs[half + i] : v * cs[i] + u * cs[half + i];
        }
        return v;
    };
    if (((nq | nk | a.dim) & 3) == 0) {
        for (int c = tid * 4; c < nq + nk; c += kPrepThreads * 4) {
            const float4 v = make_float4(value(c), value(c + 1), value(c + 2), value(c + 3));
            const int j = c < nq ? c : c - nq, d = j % a.dim;
            if (c < nq) *reinterpret_cast<float4 *>(Q + j) = v;
            else kv_put4(Kr + j - d, a.dim, d, v, a.split);
        }
    } else {
        for (int c = tid; c < nq + nk; c += kPrepThreads) {
            const int j = c < nq ? c : c - nq, d = j % a.dim;
            if (c < nq) Q[j] = value(c);
            else kv_put(Kr + j - d, a.dim, d, value(c), a.split);
        }
    }
}

/* ------------------------------------------------------------------ generic kernel */
constexpr int kGaThreads = 256, kGaKeys = 32, kGaPairs = kLmAttnPairs;

inline size_t ga_smem(int dim, int vdim) {
    return sizeof(float) * ((size_t)kGaPairs * dim + (size_t)kGaKeys * (dim + 1) + (size_t)kGaKeys * vdim +
                            (size_t)kGaPairs * vdim + kGaPairs * (kGaKeys + 1) + 4 * kGaPairs + kLmAttnSplits * kGaPairs);
}

/* grid = (tiles of 16 (row, head) pairs, KV heads, key splits) */
__global__ void __launch_bounds__(kGaThreads) lm_attn_generic_kernel(const LmAttn a, int M) {
    extern __shared__ float ga[];
    __shared__ int last_flag;
    pdl_launch_dependents();
    pdl_wait();
    const int dim = a.dim, vdim = a.vdim, group = a.heads / a.kv_heads;
    float *Q = ga, *K = Q + kGaPairs * dim, *V = K + kGaKeys * (dim + 1), *O = V + kGaKeys * vdim;
    float *S = O + kGaPairs * vdim, *mx = S + kGaPairs * (kGaKeys + 1), *den = mx + kGaPairs, *cor = den + kGaPairs,
          *wgt = cor + 2 * kGaPairs;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int g = blockIdx.y, p0 = blockIdx.x * kGaPairs;
    const int np = M * group - p0 < kGaPairs ? M * group - p0 : kGaPairs;
    const int pos0 = a.dyn->pos;
    const KeyTiles kt = key_tiles<kGaKeys>(pos0 + p0 / group, pos0 + (p0 + np - 1) / group, a.window, a.keep);
    const int S_eff = (int)gridDim.z < kt.n_tiles ? (int)gridDim.z : kt.n_tiles;
    const int sp = blockIdx.z;
    if (sp >= S_eff) return;
    const int t0 = (int)((long long)kt.n_tiles * sp / S_eff), t1 = (int)((long long)kt.n_tiles * (sp + 1) / S_eff);
    const float *Kc = lm_state(a.k, a.dyn), *Vc = lm_state(a.v, a.dyn);
    const int ldk = a.kv_heads * dim, ldv = a.kv_heads * vdim;

    for (int i = tid; i < np * dim; i += kGaThreads) {
        const int p = p0 + i / dim, d = i % dim;
        Q[i] = a.q[(size_t)(p / group) * a.heads * dim + (size_t)(g * group + p % group) * dim + d];
    }
    for (int i = tid; i < np * vdim; i += kGaThreads) O[i] = 0.0f;
    if (tid < kGaPairs) { mx[tid] = -INFINITY; den[tid] = 0.0f; }

    for (int t = t0; t < t1; t++) {
        int j0, n;
        key_tile<kGaKeys>(kt, t, &j0, &n);
        __syncthreads();
        for (int i = tid; i < n * dim; i += kGaThreads) {
            const int j = i / dim, d = i % dim;
            K[j * (dim + 1) + d] = kv_get(Kc + (size_t)lm_ring_row(a.ring, j0 + j) * ldk + g * dim, dim, d, a.split);
        }
        for (int i = tid; i < n * vdim; i += kGaThreads) {
            const int j = i / vdim, d = i % vdim;
            V[i] = kv_get(Vc + (size_t)lm_ring_row(a.ring, j0 + j) * ldv + g * vdim, vdim, d, a.split);
        }
        __syncthreads();
        for (int p = warp; p < np; p += kGaThreads / 32) {
            const int i = pos0 + (p0 + p) / group;
            float s = -INFINITY;
            if (lane < n && key_seen(i, j0 + lane, a.window, a.keep)) {
                const float *q = Q + p * dim, *k = K + lane * (dim + 1);
                float e0 = 0.0f, e1 = 0.0f, e2 = 0.0f, e3 = 0.0f;
                int d = 0;
                for (; d + 3 < dim; d += 4) {
                    e0 = fmaf(q[d], k[d], e0);
                    e1 = fmaf(q[d + 1], k[d + 1], e1);
                    e2 = fmaf(q[d + 2], k[d + 2], e2);
                    e3 = fmaf(q[d + 3], k[d + 3], e3);
                }
                for (; d < dim; d++) e0 = fmaf(q[d], k[d], e0);
                s = ((e0 + e1) + (e2 + e3)) * a.scale;
                if (a.softcap > 0.0f) s = a.softcap * tanhf(s / a.softcap);
            }
            float top = s;
#pragma unroll
            for (int o = 16; o > 0; o >>= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, o));
            const float old = mx[p], now = fmaxf(old, top);
            const float w = s > -INFINITY ? expf(s - now) : 0.0f;
            const float sum = vb_warp_sum(w);
            S[p * (kGaKeys + 1) + lane] = w;
            __syncwarp();
            if (lane == 0) {
                const float c = old > -INFINITY ? expf(old - now) : 0.0f;
                cor[p] = c;
                mx[p] = now;
                den[p] = den[p] * c + sum;
            }
        }
        __syncthreads();
        for (int i = tid; i < np * vdim; i += kGaThreads) {
            const int p = i / vdim, d = i % vdim;
            float o = O[i] * cor[p];
            const float *w = S + p * (kGaKeys + 1);
            for (int j = 0; j < n; j++) o = fmaf(w[j], V[j * vdim + d], o);
            O[i] = o;
        }
    }
    __syncthreads();

    float *po = nullptr;
    if (S_eff > 1) {
        /* several CTAs share these pairs: publish the slice, the last arrival merges in slice order */
        const int stride = vdim + 2;
        const size_t tile = (size_t)blockIdx.y * gridDim.x + blockIdx.x;
        po = a.scratch + tile * gridDim.z * kGaPairs * stride;
        float *mine = po + (size_t)sp * kGaPairs * stride;
        for (int i = tid; i < np * vdim; i += kGaThreads) mine[(i / vdim) * stride + i % vdim] = O[i];
        if (tid < np) { mine[tid * stride + vdim] = mx[tid]; mine[tid * stride + vdim + 1] = den[tid]; }
        __threadfence();
        __syncthreads();
        if (tid == 0) {
            const unsigned t = atomicAdd(&a.tickets[tile], 1u);
            last_flag = t == (unsigned)(S_eff - 1);
            if (last_flag) a.tickets[tile] = 0u;
        }
        __syncthreads();
        if (!last_flag) return;
        __threadfence();
        if (tid < np) {
            float M0 = -INFINITY, L = 0.0f;
            for (int u = 0; u < S_eff; u++) M0 = fmaxf(M0, __ldcg(po + ((size_t)u * kGaPairs + tid) * stride + vdim));
            for (int u = 0; u < S_eff; u++) {
                const float mu = __ldcg(po + ((size_t)u * kGaPairs + tid) * stride + vdim);
                const float w = mu > -INFINITY ? expf(mu - M0) : 0.0f;
                wgt[u * kGaPairs + tid] = w;
                L += w * __ldcg(po + ((size_t)u * kGaPairs + tid) * stride + vdim + 1);
            }
            den[tid] = L;
        }
        __syncthreads();
        for (int i = tid; i < np * vdim; i += kGaThreads) {
            const int p = i / vdim, d = i % vdim;
            float o = 0.0f;
            for (int u = 0; u < S_eff; u++) o = fmaf(wgt[u * kGaPairs + p], __ldcg(po + ((size_t)u * kGaPairs + p) * stride + d), o);
            O[i] = o;
        }
        __syncthreads();
    }
    for (int i = tid; i < np * vdim; i += kGaThreads) {
        const int p = i / vdim, d = i % vdim, P = p0 + p;
        lm_put(a.out, P / group, (g * group + P % group) * vdim + d, O[i] / den[p]);
    }
}

/* ------------------------------------------------------------------ one token */
constexpr int kSaThreads = 512, kSaWarps = 16;

/* grid = (key splits, KV heads). Every CTA sums the squares of the whole q and k projection itself
 * (a few L2 reads instead of another launch), norms and rotates its own heads, and attends over its
 * share of the visible keys: a warp serves one head of the group on one of 16 / (heads of the group)
 * subsets of the keys, KP keys in flight, a lane four dimensions per step. The last split owns the
 * new token and appends it. ND, NV: 128-wide steps of the key and value sizes. */
template <int ND, int NV, int KP, bool SPLIT>
__global__ void __launch_bounds__(kSaThreads) lm_attn_step_kernel(const LmAttn a, int lanes_h) {
    extern __shared__ __align__(16) float sa[];
    __shared__ float red[2][kSaWarps], sub_m[kSaWarps], sub_l[kSaWarps], wgt[kLmAttnSplits * kSaWarps];
    __shared__ int last_flag;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int dim = a.dim, vdim = a.vdim, group = a.heads / a.kv_heads, half = a.rot / 2;
    const int nq = a.heads * dim, nk = a.kv_heads * dim, nv = a.kv_heads * vdim;
    float *raw = sa;                                       /* [group * dim] own q, then [dim] own k */
    float *qs = raw + (group + 1) * dim;                   /* [group][dim] */
    float *os = qs + group * dim;                          /* [16 warps][vdim] */
    float *cs = os + kSaWarps * vdim;                      /* [rot] */
    pdl_launch_dependents();
    pdl_wait();
    const int sp = blockIdx.x, g = blockIdx.y;
    const int pos = a.dyn->pos;
    /* visible keys in order: the kept ones, then the window */
    const int n_keep = a.window > 0 ? (a.keep < pos + 1 ? a.keep : pos + 1) : 0;
    const int w0 = a.window > 0 ? (pos - a.window + 1 > n_keep ? pos - a.window + 1 : n_keep) : 0;
    const int n_keys = n_keep + (pos + 1 - w0);
    int S = (n_keys + 31) / 32;
    if (S > (int)gridDim.x) S = gridDim.x;
    if (sp >= S) return;
    const int x0 = (int)((long long)n_keys * sp / S), x1 = (int)((long long)n_keys * (sp + 1) / S);
    const bool writer = sp == S - 1;

    float sq = 0.0f, sk = 0.0f;
    const int own0 = g * group * dim, own1 = own0 + group * dim, k0 = nq + g * dim, k1 = k0 + dim;
    for (int c = tid * 4; c < nq + nk; c += kSaThreads * 4) {
        const float4 v = lm_sum4(a.qkv, 0, c);
        const float ss = v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        if (c < nq) sq += ss; else sk += ss;
        if (c >= own0 && c < own1) *reinterpret_cast<float4 *>(raw + c - own0) = v;
        else if (c >= k0 && c < k1) *reinterpret_cast<float4 *>(raw + group * dim + c - k0) = v;
    }
    float *Kc = lm_state(a.k, a.dyn) + g * dim, *Vc = lm_state(a.v, a.dyn) + g * vdim;
    const size_t new_row = (size_t)lm_ring_row(a.ring, pos);
    if (writer)
        for (int c = tid; c < vdim; c += kSaThreads) kv_put(Vc + new_row * nv, vdim, c, lm_sum_batch(a.qkv, 0, nq + nk + g * vdim + c), SPLIT);
    for (int i = tid; i < half; i += kSaThreads) {
        lm_angle(pos, a.freq[i], a.freq[half + i], a.mag, &cs[i], &cs[half + i]);
    }
    sq = vb_warp_sum(sq);
    sk = vb_warp_sum(sk);
    if (lane == 0) { red[0][warp] = sq; red[1][warp] = sk; }
    __syncthreads();
    sq = sk = 0.0f;
#pragma unroll
    for (int w = 0; w < kSaWarps; w++) { sq += red[0][w]; sk += red[1][w]; }
    const float rq = 1.0f / sqrtf(sq / (float)nq + a.eps), rk = 1.0f / sqrtf(sk / (float)nk + a.eps);
    const int total = (writer ? group + 1 : group) * dim;
    for (int i = tid; i < total; i += kSaThreads) {
        const bool isq = i < group * dim;
        const int d = i % dim;
        const float *gain = isq ? a.q_gain + own0 + i : a.k_gain + g * dim + d;
        const float r = isq ? rq : rk;
        float v = raw[i] * r * __ldg(gain);
        if (d < a.rot) {
            const int j = d < half ? d : d - half, other = d < half ? half : -half;
            const float u = raw[i + other] * r * __ldg(gain + other);
            v = d < half ? v * cs[j] - u * cs[half + j] : v * cs[j] + u * cs[half + j];
        }
        if (isq) qs[i] = v;
        else kv_put(Kc + new_row * nk, dim, d, v, SPLIT);
    }
    __syncthreads();          /* the appended row is visible to this CTA */

    const int hh = warp % lanes_h, sub = warp / lanes_h, subs = kSaWarps / lanes_h;
    float mx = -INFINITY, den = 0.0f, o[NV][4];
#pragma unroll
    for (int i = 0; i < NV; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    if (hh < group) {
        float4 q[ND];
#pragma unroll
        for (int i = 0; i < ND; i++) {
            const int d = i * 128 + lane * 4;
            q[i] = d < dim ? *reinterpret_cast<const float4 *>(qs + hh * dim + d) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        const int first = w0 > a.ring.keep ? (w0 - a.ring.keep) % a.ring.ring : 0;      /* ring place of the window's first key */
        for (int xb = x0 + sub; xb < x1; xb += KP * subs) {
            /* every load of the pass is requested unconditionally (beyond the range: the last key again), so that
             * they are all in flight together */
            float4 kk[KP][ND], vv[KP][NV];
#pragma unroll
            for (int u = 0; u < KP; u++) {
                int x = xb + u * subs;
                x = x < x1 ? x : x1 - 1;
                int r = first + x - n_keep;
                r = x < n_keep ? x : a.ring.keep + (r < a.ring.ring ? r : r - a.ring.ring);
#pragma unroll
                for (int i = 0; i < ND; i++) {
                    const int d = i * 128 + lane * 4;
                    kk[u][i] = kv_get4<SPLIT>(Kc + (size_t)r * nk, dim, d < dim ? d : 0);
                }
#pragma unroll
                for (int i = 0; i < NV; i++) {
                    const int d = i * 128 + lane * 4;
                    vv[u][i] = kv_get4<SPLIT>(Vc + (size_t)r * nv, vdim, d < vdim ? d : 0);
                }
            }
            float s[KP];
#pragma unroll
            for (int u = 0; u < KP; u++) {
                s[u] = 0.0f;
#pragma unroll
                for (int i = 0; i < ND; i++)
                    s[u] += q[i].x * kk[u][i].x + q[i].y * kk[u][i].y + q[i].z * kk[u][i].z + q[i].w * kk[u][i].w;
            }
            /* a lane ends up with the score of one of the pass's keys (32 / KP lanes share one) */
            constexpr int kShare = 32 / KP;
            vb_warp_multi_sum<KP>(s, lane);
            float sc = s[0] * a.scale;
            if (a.softcap > 0.0f) sc = a.softcap * tanhf(sc / a.softcap);
            if (xb + (lane / kShare) * subs >= x1) sc = -INFINITY;
            float top = sc;
#pragma unroll
            for (int off = kShare; off < 32; off <<= 1) top = fmaxf(top, __shfl_xor_sync(0xffffffffu, top, off));
            top = fmaxf(top, mx);                         /* the first key of a pass is always there: finite */
            const float c = expf(mx - top), w = expf(sc - top);
            mx = top;
            den = den * c + w;                            /* this lane's key only; added up at the end */
#pragma unroll
            for (int i = 0; i < NV; i++) { o[i][0] *= c; o[i][1] *= c; o[i][2] *= c; o[i][3] *= c; }
#pragma unroll
            for (int u = 0; u < KP; u++) {
                const float wu = __shfl_sync(0xffffffffu, w, u * kShare);
#pragma unroll
                for (int i = 0; i < NV; i++) {
                    o[i][0] = fmaf(wu, vv[u][i].x, o[i][0]);
                    o[i][1] = fmaf(wu, vv[u][i].y, o[i][1]);
                    o[i][2] = fmaf(wu, vv[u][i].z, o[i][2]);
                    o[i][3] = fmaf(wu, vv[u][i].w, o[i][3]);
                }
            }
        }
#pragma unroll
        for (int off = 32 / KP; off < 32; off <<= 1) den += __shfl_xor_sync(0xffffffffu, den, off);
    }
#pragma unroll
    for (int i = 0; i < NV; i++) {
        const int d = i * 128 + lane * 4;
        if (d < vdim) *reinterpret_cast<float4 *>(os + warp * vdim + d) = make_float4(o[i][0], o[i][1], o[i][2], o[i][3]);
    }
    if (lane == 0) { sub_m[warp] = mx; sub_l[warp] = den; }
    __syncthreads();
    /* merge the key subsets of every head, in order */
    const int stride = vdim + 2;
    float *po = a.scratch + (size_t)g * gridDim.x * group * stride;            /* [split][head][vdim + 2] */
    for (int i = tid; i < group * vdim; i += kSaThreads) {
        const int hd = i / vdim, d = i % vdim;
        float M0 = -INFINITY, L = 0.0f, O = 0.0f;
        for (int u = 0; u < subs; u++) M0 = fmaxf(M0, sub_m[u * lanes_h + hd]);
        for (int u = 0; u < subs; u++) {
            const int w = u * lanes_h + hd;
            const float f = sub_m[w] > -INFINITY ? expf(sub_m[w] - M0) : 0.0f;
            L = fmaf(sub_l[w], f, L);
            O = fmaf(os[w * vdim + d], f, O);
        }
        if (S == 1) {
            lm_put(a.out, 0, (g * group + hd) * vdim + d, O / L);
        } else {
            float *mine = po + ((size_t)sp * group + hd) * stride;
            mine[d] = O;
            if (d == 0) { mine[vdim] = M0; mine[vdim + 1] = L; }
        }
    }
    if (S == 1) return;
    __threadfence();
    __syncthreads();
    if (tid == 0) {
        const unsigned t = atomicAdd(&a.tickets[g], 1u);
        last_flag = t == (unsigned)(S - 1);
        if (last_flag) a.tickets[g] = 0u;
    }
    __syncthreads();
    if (!last_flag) return;
    __threadfence();
    /* weights of the slices per head, then the slices in order */
    if (tid < group) {
        float m[kLmAttnSplits], M0 = -INFINITY, L = 0.0f;
#pragma unroll
        for (int u = 0; u < kLmAttnSplits; u++) m[u] = u < S ? __ldcg(po + ((size_t)u * group + tid) * stride + vdim) : -INFINITY;
#pragma unroll
        for (int u = 0; u < kLmAttnSplits; u++) M0 = fmaxf(M0, m[u]);
#pragma unroll
        for (int u = 0; u < kLmAttnSplits; u++)
            if (u < S) {
                const float f = expf(m[u] - M0);
                L = fmaf(__ldcg(po + ((size_t)u * group + tid) * stride + vdim + 1), f, L);
                wgt[u * kSaWarps + tid] = f;
            }
        sub_l[tid] = L;
    }
    __syncthreads();
    for (int i = tid; i < group * vdim; i += kSaThreads) {
        const int hd = i / vdim, d = i % vdim;
        float t[kLmAttnSplits], O = 0.0f;
#pragma unroll
        for (int u = 0; u < kLmAttnSplits; u++) t[u] = u < S ? __ldcg(po + ((size_t)u * group + hd) * stride + d) : 0.0f;
#pragma unroll
        for (int u = 0; u < kLmAttnSplits; u++)
            if (u < S) O = fmaf(t[u], wgt[u * kSaWarps + hd], O);
        lm_put(a.out, 0, (g * group + hd) * vdim + d, O / sub_l[hd]);
    }
}

inline size_t step_smem(const LmAttn &a) {
    const int group = a.heads / a.kv_heads;
    return sizeof(float) * ((size_t)(2 * group + 1) * a.dim + (size_t)kSaWarps * a.vdim + a.rot + 4);
}

template <int ND, int NV, int KP, bool SPLIT>
int launch_attn_step(const LmAttn &a, int splits, int lanes_h, cudaStream_t st) {
    const size_t smem = step_smem(a);
    static size_t set = 48 * 1024;
    if (smem > set) {
        if (cudaFuncSetAttribute(lm_attn_step_kernel<ND, NV, KP, SPLIT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        set = smem;
    }
    return ok(launch_pdl(lm_attn_step_kernel<ND, NV, KP, SPLIT>, dim3(splits, a.kv_heads), dim3(kSaThreads), smem, st, a, lanes_h));
}

/* ------------------------------------------------------------------ prompts on the warp-level tensor cores */
constexpr int kMaThreads = 256, kMaWarps = 8, kMaKeys = 32;

/* Requests 32 keys of one KV head: the high and low halves of the cache rows, 16 bytes per copy,
 * straight into the swizzled tiles. What lies beyond the head's size in a tile is not touched. */
template <int STEPS>
VB_DEVINL void request_tile(unsigned char *hi_t, const float *cache, int ld, int col0, int size, int j0, int n, const LmRing &ring) {
    const int per = size / 8;                           /* chunks of a plane */
    for (int i = threadIdx.x; i < n * 2 * per; i += kMaThreads) {
        const int key = i / (2 * per), f = i % (2 * per), plane = f >= per ? 1 : 0, chunk = f - plane * per;
        const uint16_t *src = reinterpret_cast<const uint16_t *>(cache + (size_t)lm_ring_row(ring, j0 + key) * ld + col0) + f * 8;
        lm_cp16(hi_t + plane * (kMaKeys * STEPS * 32) + tile_off<STEPS>(key, chunk), src);
    }
}
/* The same out of keys and values that were read out of a latent: a head's own columns from the written-out
 * rows, then `shared` columns (the key part all heads have in common) from the latent's cache row. */
template <int STEPS>
VB_DEVINL void request_wide(unsigned char *hi_t, const LmWide &w, int col0, int size, int shared, int j0, int n, const LmRing &ring) {
    const int own = size / 8, per = own + shared / 8, row = w.rank + w.rot_dim;
    for (int i = threadIdx.x; i < n * 2 * per; i += kMaThreads) {
        const int key = i / (2 * per), f = i % (2 * per), plane = f >= per ? 1 : 0, chunk = f - plane * per;
        const uint16_t *src;
        if (chunk < own) src = w.kv + plane * w.plane + (size_t)(j0 + key - w.first) * w.ld + col0 + chunk * 8;
        else src = reinterpret_cast<const uint16_t *>(w.cache + (size_t)lm_ring_row(ring, j0 + key) * row) + plane * row + w.rank + (chunk - own) * 8;
        lm_cp16(hi_t + plane * (kMaKeys * STEPS * 32) + tile_off<STEPS>(key, chunk), src);
    }
}

struct LmNotWide {};
template <bool WIDE> struct LmWideSel { using type = LmNotWide; };
template <> struct LmWideSel<true> { using type = LmWide; };

/* cap * tanh(x / cap), the hyperbolic tangent through one exponential (absolute error about 1e-7 of cap) */
VB_DEVINL float soft_cap(float x, float cap, float two_over_cap) {
    return cap - 2.0f * cap * __fdividef(1.0f, 1.0f + __expf(x * two_over_cap));
}

/* WIDE: every head has keys and values of its own, read out of a latent (LmWide).
 * A CTA serves one KV head; each of its eight warps owns 16 query rows of one query head of the
 * group (consecutive (row block, head) tiles), so that the staged keys are shared by up to eight
 * warps. Every product a.b is taken as a_hi.b_hi + a_hi.b_lo + a_lo.b_hi, accumulated in fp32;
 * scores, softcap, weights and the running maximum are fp32. DK, DV: 16-wide steps of the key
 * and value sizes (padded with zeros). */
template <int DK, int DV, bool WIDE>
__global__ void __launch_bounds__(kMaThreads) lm_attn_mma_kernel(const LmAttn a, const typename LmWideSel<WIDE>::type wide, int M) {
    extern __shared__ __align__(128) unsigned char ma_tiles[];
    /* two buffers of K high, K low, V high, V low */
    constexpr int kTileK = kMaKeys * DK * 32, kTileV = kMaKeys * DV * 32, kBuf = 2 * (kTileK + kTileV);
    pdl_launch_dependents();
    for (int i = threadIdx.x; i < 2 * kBuf / 16; i += kMaThreads) reinterpret_cast<uint4 *>(ma_tiles)[i] = make_uint4(0u, 0u, 0u, 0u);
    pdl_wait();
    __syncthreads();
    const int group = a.heads / a.kv_heads, g = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    const int n_tiles_q = (M + 15) / 16 * group;
    /* the latest rows see the most keys: they go first */
    const int T0 = ((int)gridDim.x - 1 - (int)blockIdx.x) * kMaWarps, T1 = T0 + kMaWarps < n_tiles_q ? T0 + kMaWarps : n_tiles_q;
    const int T = T0 + warp;
    const bool active = T < T1;
    const int r0 = active ? T / group * 16 : 0, h = g * group + (active ? T % group : 0);
    const int pos0 = a.dyn->pos;
    const int rowA = r0 + gq, rowB = rowA + 8;
    const bool validA = active && rowA < M, validB = active && rowB < M;
    const int iA = pos0 + rowA, iB = pos0 + rowB;
    const int last_row = T1 > T0 ? ((T1 - 1) / group * 16 + 15 < M - 1 ? (T1 - 1) / group * 16 + 15 : M - 1) : 0;
    const KeyTiles kt = key_tiles<kMaKeys>(pos0 + T0 / group * 16, pos0 + last_row, a.window, a.keep);
    const int w_imin = pos0 + r0, w_imax = pos0 + (r0 + 15 < M - 1 ? r0 + 15 : M - 1);
    const float *Kc = nullptr, *Vc = nullptr;
    if constexpr (!WIDE) { Kc = lm_state(a.k, a.dyn); Vc = lm_state(a.v, a.dyn); }
    const int ldk = a.kv_heads * a.dim, ldv = a.kv_heads * a.vdim;
    typename LmWideSel<WIDE>::type lw = wide;
    if constexpr (WIDE) lw.cache += (size_t)a.dyn->slot * lw.slab;

    /* Q as A fragments: (row A, k 2t..), (row B, k 2t..), (row A, k 8 + 2t..), (row B, k 8 + 2t..) */
    uint32_t qh[DK][4], ql[DK][4];
#pragma unroll
    for (int ks = 0; ks < DK; ks++)
#pragma unroll
        for (int hf = 0; hf < 2; hf++)
#pragma unroll
            for (int rr = 0; rr < 2; rr++) {
                const int d = ks * 16 + hf * 8 + 2 * tq;
                const bool v = rr ? validB : validA;
                float q0 = 0.0f, q1 = 0.0f;
                if constexpr (WIDE) {
                    if (v && d < a.dim) {          /* dim is a multiple of 8: d and d + 1 are a rotated pair or neither is */
                        const int row = rr ? rowB : rowA, i = (d - (a.dim - wide.rot_dim)) / 2, half = a.rot / 2;
                        const float2 u = lm_sum2(wide.q, row, h * a.dim + d);
                        q0 = u.x; q1 = u.y;
                        if (d >= a.dim - wide.rot_dim && i < half) {
                            const float c = wide.cs[(size_t)row * a.rot + i], s = wide.cs[(size_t)row * a.rot + half + i];
                            q0 = u.x * c - u.y * s;
                            q1 = u.y * c + u.x * s;
                        }
                    }
                } else {
                    const float *q = a.q + (size_t)(rr ? rowB : rowA) * a.heads * a.dim + (size_t)h * a.dim + d;
                    if (v && d < a.dim) q0 = q[0];
                    if (v && d + 1 < a.dim) q1 = q[1];
                }
                uint32_t h0, l0, h1, l1;
                hilo(q0, h0, l0);
                hilo(q1, h1, l1);
                qh[ks][hf * 2 + rr] = h0 | (h1 << 16);
                ql[ks][hf * 2 + rr] = l0 | (l1 << 16);
            }
    float o[2 * DV][4];
#pragma unroll
    for (int i = 0; i < 2 * DV; i++) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.0f;
    float mA = -INFINITY, mB = -INFINITY, lA = 0.0f, lB = 0.0f;
    const uint32_t smem0 = vb_smem_u32(ma_tiles);
    const int mat = lane >> 3, mr = lane & 7;
    const float two_over_cap = a.softcap > 0.0f ? 2.0f / a.softcap : 0.0f;
    auto request = [&](int t) {
        int j0, n;
        key_tile<kMaKeys>(kt, t, &j0, &n);
        unsigned char *b = ma_tiles + (t & 1) * kBuf;
        if constexpr (WIDE) {
            request_wide<DK>(b, lw, g * (a.dim - lw.rot_dim), a.dim - lw.rot_dim, lw.rot_dim, j0, n, a.ring);
            request_wide<DV>(b + 2 * kTileK, lw, lw.v0 + g * a.vdim, a.vdim, 0, j0, n, a.ring);
        } else {
            request_tile<DK>(b, Kc, ldk, g * a.dim, a.dim, j0, n, a.ring);
            request_tile<DV>(b + 2 * kTileK, Vc, ldv, g * a.vdim, a.vdim, j0, n, a.ring);
        }
        lm_cp_commit();
    };
    if (kt.n_tiles > 0) request(0);

    for (int t = 0; t < kt.n_tiles; t++) {
        int j0, n;
        key_tile<kMaKeys>(kt, t, &j0, &n);
        lm_cp_wait_all();
        __syncthreads();                               /* this buffer is complete, the other one is free */
        if (t + 1 < kt.n_tiles) request(t + 1);
        const uint32_t sKh = smem0 + (uint32_t)((t & 1) * kBuf), sKl = sKh + kTileK, sVh = sKl + kTileK, sVl = sVh + kTileV;
        /* nothing of this tile for this warp's rows: later than all of them, or behind every window and not kept */
        if (!active || j0 > w_imax || (a.window > 0 && w_imin - (j0 + n - 1) >= a.window && j0 >= a.keep)) continue;

        float s[4][4];
#pragma unroll
        for (int i = 0; i < 4; i++) s[i][0] = s[i][1] = s[i][2] = s[i][3] = 0.0f;
#pragma unroll
        for (int ks = 0; ks < DK; ks++) {
#pragma unroll
            for (int kp = 0; kp < 2; kp++) {           /* 16 keys each */
                const uint32_t off = tile_off<DK>(kp * 16 + (mat >> 1) * 8 + mr, ks * 2 + (mat & 1));
                uint32_t bh[4], bl[4];
                ldsm(bh, sKh + off);
                ldsm(bl, sKl + off);
                mma_bf16(s[kp * 2], qh[ks], bh[0], bh[1]);
                mma_bf16(s[kp * 2 + 1], qh[ks], bh[2], bh[3]);
                mma_bf16(s[kp * 2], qh[ks], bl[0], bl[1]);
                mma_bf16(s[kp * 2 + 1], qh[ks], bl[2], bl[3]);
                mma_bf16(s[kp * 2], ql[ks], bh[0], bh[1]);
                mma_bf16(s[kp * 2 + 1], ql[ks], bh[2], bh[3]);
            }
        }
        float tA = -INFINITY, tB = -INFINITY;
#pragma unroll
        for (int nt = 0; nt < 4; nt++)
#pragma unroll
            for (int c = 0; c < 4; c++) {
                const int key = nt * 8 + 2 * tq + (c & 1);
                float v = s[nt][c] * a.scale;
                if (a.softcap > 0.0f) v = soft_cap(v, a.softcap, two_over_cap);
                if (key >= n || !key_seen(c < 2 ? iA : iB, j0 + key, a.window, a.keep)) v = -INFINITY;
                s[nt][c] = v;
                if (c < 2) tA = fmaxf(tA, v); else tB = fmaxf(tB, v);
            }
        tA = fmaxf(tA, __shfl_xor_sync(0xffffffffu, tA, 1));
        tA = fmaxf(tA, __shfl_xor_sync(0xffffffffu, tA, 2));
        tB = fmaxf(tB, __shfl_xor_sync(0xffffffffu, tB, 1));
        tB = fmaxf(tB, __shfl_xor_sync(0xffffffffu, tB, 2));
        /* a row that has seen no key yet keeps a finite reference, so that every weight below is exp(-inf) = 0 */
        const float nA = fmaxf(mA, tA), nB = fmaxf(mB, tB);
        const float fA = nA > -INFINITY ? nA : 0.0f, fB = nB > -INFINITY ? nB : 0.0f;
        const float cA = expf(mA - fA), cB = expf(mB - fB);
        mA = nA; mB = nB;
        float sumA = 0.0f, sumB = 0.0f;
        uint32_t ph[2][4], pl[2][4];
#pragma unroll
        for (int nt = 0; nt < 4; nt++) {
            const float p0 = expf(s[nt][0] - fA), p1 = expf(s[nt][1] - fA), p2 = expf(s[nt][2] - fB), p3 = expf(s[nt][3] - fB);
            sumA += p0 + p1;
            sumB += p2 + p3;
            uint32_t h0, l0, h1, l1;
            hilo(p0, h0, l0); hilo(p1, h1, l1);
            ph[nt >> 1][(nt & 1) * 2] = h0 | (h1 << 16);
            pl[nt >> 1][(nt & 1) * 2] = l0 | (l1 << 16);
            hilo(p2, h0, l0); hilo(p3, h1, l1);
            ph[nt >> 1][(nt & 1) * 2 + 1] = h0 | (h1 << 16);
            pl[nt >> 1][(nt & 1) * 2 + 1] = l0 | (l1 << 16);
        }
        lA = lA * cA + sumA;
        lB = lB * cB + sumB;
#pragma unroll
        for (int i = 0; i < 2 * DV; i++) { o[i][0] *= cA; o[i][1] *= cA; o[i][2] *= cB; o[i][3] *= cB; }
#pragma unroll
        for (int dp = 0; dp < DV; dp++) {
#pragma unroll
            for (int kp = 0; kp < 2; kp++) {
                const uint32_t off = tile_off<DV>(kp * 16 + (mat & 1) * 8 + mr, dp * 2 + (mat >> 1));
                uint32_t vh[4], vl[4];
                ldsm_t(vh, sVh + off);
                ldsm_t(vl, sVl + off);
                mma_bf16(o[2 * dp], ph[kp], vh[0], vh[1]);
                mma_bf16(o[2 * dp + 1], ph[kp], vh[2], vh[3]);
                mma_bf16(o[2 * dp], ph[kp], vl[0], vl[1]);
                mma_bf16(o[2 * dp + 1], ph[kp], vl[2], vl[3]);
                mma_bf16(o[2 * dp], pl[kp], vh[0], vh[1]);
                mma_bf16(o[2 * dp + 1], pl[kp], vh[2], vh[3]);
            }
        }
    }
    lA += __shfl_xor_sync(0xffffffffu, lA, 1);
    lA += __shfl_xor_sync(0xffffffffu, lA, 2);
    lB += __shfl_xor_sync(0xffffffffu, lB, 1);
    lB += __shfl_xor_sync(0xffffffffu, lB, 2);
    float rA = 1.0f / lA, rB = 1.0f / lB;
    if constexpr (WIDE) {
        if (validA) rA *= wide.gate[(size_t)rowA * a.heads + h];
        if (validB) rB *= wide.gate[(size_t)rowB * a.heads + h];
    }
#pragma unroll
    for (int nt = 0; nt < 2 * DV; nt++)
#pragma unroll
        for (int u = 0; u < 2; u++) {
            const int d = nt * 8 + 2 * tq + u;
            if (d >= a.vdim) continue;
            if (validA) lm_put(a.out, rowA, h * a.vdim + d, o[nt][u] * rA);
            if (validB) lm_put(a.out, rowB, h * a.vdim + d, o[nt][2 + u] * rB);
        }
}

template <int DK, int DV, bool WIDE>
int launch_mma(const LmAttn &a, const typename LmWideSel<WIDE>::type &wide, int M, cudaStream_t st) {
    constexpr size_t smem = (size_t)2 * kMaKeys * 64 * (DK + DV);
    static bool attr = false;
    if (!attr) {
        if (cudaFuncSetAttribute(lm_attn_mma_kernel<DK, DV, WIDE>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        attr = true;
    }
    const int tiles = (M + 15) / 16 * (a.heads / a.kv_heads);
    return ok(launch_pdl(lm_attn_mma_kernel<DK, DV, WIDE>, dim3((tiles + kMaWarps - 1) / kMaWarps, a.kv_heads), dim3(kMaThreads), smem, st, a, wide, M));
}

constexpr int kSplitBudget = 296;        /* two CTAs per SM */
constexpr int kStepCtas = 148;           /* one-token kernel: one CTA per SM */

} // namespace

size_t lm_attn_scratch_floats(int heads, int kv_heads, int vdim) {
    (void)heads; (void)kv_heads;
    return (size_t)kSplitBudget * kLmAttnPairs * (vdim + 2);
}
int lm_attn_ticket_count(int heads, int kv_heads) {
    (void)heads; (void)kv_heads;
    return kSplitBudget;
}

int lm_attn_prepare(const LmAttn &a, int M, cudaStream_t st) {
    const size_t smem = sizeof(float) * ((size_t)(a.heads + a.kv_heads) * a.dim + a.rot);
    if (smem > 200 * 1024) return -1;
    static size_t set = 48 * 1024;
    if (smem > set) {
        if (cudaFuncSetAttribute(lm_attn_prepare_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        set = smem;
    }
    return ok(launch_pdl(lm_attn_prepare_kernel, dim3(M), dim3(kPrepThreads), smem, st, a));
}

int lm_attn_generic(const LmAttn &a, int M, cudaStream_t st) {
    const size_t smem = ga_smem(a.dim, a.vdim);
    if (smem > 200 * 1024) return -1;
    static size_t set = 48 * 1024;
    if (smem > set) {
        if (cudaFuncSetAttribute(lm_attn_generic_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        set = smem;
    }
    const int tiles = (M * (a.heads / a.kv_heads) + kGaPairs - 1) / kGaPairs;
    int splits = kSplitBudget / (tiles * a.kv_heads);
    splits = splits < 1 ? 1 : splits > kLmAttnSplits ? kLmAttnSplits : splits;
    return ok(launch_pdl(lm_attn_generic_kernel, dim3(tiles, a.kv_heads, splits), dim3(kGaThreads), smem, st, a, M));
}

bool lm_attn_mma_ok(int dim, int vdim) { return dim <= 128 && vdim <= 128 && dim % 8 == 0 && vdim % 8 == 0; }

int lm_attn_mma(const LmAttn &a, int M, cudaStream_t st) {
    const bool k4 = a.dim <= 64, v4 = a.vdim <= 64;
    const LmNotWide w;
    if (k4) return v4 ? launch_mma<4, 4, false>(a, w, M, st) : launch_mma<4, 8, false>(a, w, M, st);
    return v4 ? launch_mma<8, 4, false>(a, w, M, st) : launch_mma<8, 8, false>(a, w, M, st);
}

bool lm_attn_wide_ok(int plain, int rot_dim, int vdim) {
    return plain + rot_dim <= 192 && vdim <= 128 && plain % 8 == 0 && rot_dim % 8 == 0 && vdim % 8 == 0;
}

int lm_attn_wide(const LmAttn &a, const LmWide &w, int M, cudaStream_t st) {
    const bool v4 = a.vdim <= 64;
    if (a.dim <= 64) return v4 ? launch_mma<4, 4, true>(a, w, M, st) : launch_mma<4, 8, true>(a, w, M, st);
    if (a.dim <= 128) return v4 ? launch_mma<8, 4, true>(a, w, M, st) : launch_mma<8, 8, true>(a, w, M, st);
    return v4 ? launch_mma<12, 4, true>(a, w, M, st) : launch_mma<12, 8, true>(a, w, M, st);
}

bool lm_attn_step_ok(const LmAttn &a) {
    return a.heads / a.kv_heads <= kSaWarps && a.kv_heads <= kSplitBudget && a.dim % 4 == 0 && a.vdim % 4 == 0 && a.dim <= 256 &&
           a.vdim <= 256;
}

int lm_attn_step(const LmAttn &a, cudaStream_t st) {
    const int group = a.heads / a.kv_heads;
    int lanes_h = 1;
    while (lanes_h < group) lanes_h *= 2;
    int splits = kStepCtas / a.kv_heads;
    splits = splits < 1 ? 1 : splits > kLmAttnSplits ? kLmAttnSplits : splits;
    if (a.split) return launch_attn_step<1, 1, 8, true>(a, splits, lanes_h, st);      /* sizes up to 128 */
    if (a.dim <= 128 && a.vdim <= 128) return launch_attn_step<1, 1, 8, false>(a, splits, lanes_h, st);
    return launch_attn_step<2, 2, 4, false>(a, splits, lanes_h, st);
}

} // namespace vb
