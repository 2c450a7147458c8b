/*
 * vb_lm_moe.cu - decoder language models: feed-forwards of many small experts, of which a token uses
 * a few (chosen by the router in the mixer's preparation kernel, weighted in the residual kernel).
 *
 *   few rows    a warp multiplies four weight rows of a chosen expert, straight from the tiles the
 *               tensor cores use, in fp32
 *   many rows   tokens are sorted by expert into blocks of 128 rows (plan, gather); the two products
 *               are grouped GEMMs on the tensor cores (tc_gemm_grouped), or fp32 ones in the 32-bit
 *               mode
 */
#include "vb_lm_kernels.cuh"
#include "vb_tc.cuh"

namespace vb {

namespace {

inline int ok(cudaError_t e) { return e == cudaSuccess ? 0 : -1; }

constexpr int kMfThreads = 256, kMfRows = 32;      /* a CTA multiplies 32 weight rows, a warp four */
constexpr int kMfPre = 8;

VB_DEVINL float dot8(const uint4 &w, const float *x) {
    const float4 a = *reinterpret_cast<const float4 *>(x), b = *reinterpret_cast<const float4 *>(x + 4);
    float v = vb_bf16_lo(w.x) * a.x;
    v = fmaf(vb_bf16_hi(w.x), a.y, v);
    v = fmaf(vb_bf16_lo(w.y), a.z, v);
    v = fmaf(vb_bf16_hi(w.y), a.w, v);
    v = fmaf(vb_bf16_lo(w.z), b.x, v);
    v = fmaf(vb_bf16_hi(w.z), b.y, v);
    v = fmaf(vb_bf16_lo(w.w), b.z, v);
    return fmaf(vb_bf16_hi(w.w), b.w, v);
}

/* act[choice][f] = max(W_up x, 0)^2 (DOWN: y[choice][n] = W_down act[choice]) of the expert each choice names.
 * grid = (32-row blocks, choices) */
template <bool DOWN>
__global__ void __launch_bounds__(kMfThreads) lm_moe_few_kernel(const LmMoe a) {
    extern __shared__ __align__(16) float xs[];              /* the row, padded to whole 64-column blocks */
    pdl_launch_dependents();
    pdl_wait();
    const int choice = blockIdx.y, m = choice / a.top, tid = threadIdx.x, lane = tid & 31;
    const int expert = a.chosen[choice];
    const LmWeight &W = DOWN ? a.down : a.up;
    const int N = DOWN ? a.width : a.ff, kblocks = W.Kp >> 6, c0 = (lane & 7) * 8;
    const int n = blockIdx.x * kMfRows + (tid >> 5) * 4 + (lane >> 3);
    const int row = expert * ((N + 127) / 128 * 128) + (n < N ? n : N - 1);
    /* the first weights are on their way while the row is put together */
    uint4 pre[kMfPre];
#pragma unroll
    for (int i = 0; i < kMfPre; i++)
        pre[i] = i < kblocks ? __ldg(reinterpret_cast<const uint4 *>(lm_weight_row(W, row, i) + c0)) : make_uint4(0u, 0u, 0u, 0u);
    if (DOWN) {
        for (int c = tid; c < W.Kp; c += kMfThreads) xs[c] = c < a.ff ? __ldcg(a.act + (size_t)choice * a.act_ld + c) : 0.0f;
    } else if (a.x.rows) {
        for (int c = tid; c < W.Kp; c += kMfThreads) xs[c] = __ldcg(a.x.rows + (size_t)m * a.x.ld + c);
    } else {
        const size_t term = (size_t)a.x.rows_pad * a.x.ld;
        for (int c = tid * 4; c < W.Kp; c += kMfThreads * 4) {
            float v[4] = {};
            for (int t = a.x.n_terms - 1; t >= 0; t--) {
                const uint2 u = __ldcg(reinterpret_cast<const uint2 *>(a.x.terms + t * term + (size_t)m * a.x.ld + c));
                v[0] += vb_bf16_lo(u.x); v[1] += vb_bf16_hi(u.x); v[2] += vb_bf16_lo(u.y); v[3] += vb_bf16_hi(u.y);
            }
            *reinterpret_cast<float4 *>(xs + c) = make_float4(v[0], v[1], v[2], v[3]);
        }
    }
    __syncthreads();
    float acc = 0.0f;
    for (int k0 = 0; k0 < kblocks; k0 += kMfPre) {
        uint4 nxt[kMfPre];
#pragma unroll
        for (int i = 0; i < kMfPre; i++) {
            const int kb = k0 + kMfPre + i;
            nxt[i] = kb < kblocks ? __ldg(reinterpret_cast<const uint4 *>(lm_weight_row(W, row, kb) + c0)) : make_uint4(0u, 0u, 0u, 0u);
        }
#pragma unroll
        for (int i = 0; i < kMfPre; i++)
            if (k0 + i < kblocks) acc += dot8(pre[i], xs + (k0 + i) * 64 + c0);
#pragma unroll
        for (int i = 0; i < kMfPre; i++) pre[i] = nxt[i];
    }
#pragma unroll
    for (int o = 4; o > 0; o >>= 1) acc += __shfl_xor_sync(0xffffffffu, acc, o);
    if ((lane & 7) == 0 && n < N) {
        if (DOWN) {
            a.y[(size_t)choice * a.y_ld + n] = acc;
        } else {
            acc = fmaxf(acc, 0.0f);
            a.act[(size_t)choice * a.act_ld + n] = acc * acc;
        }
    }
    if (DOWN && blockIdx.x == 0 && tid == 0) a.at[choice] = choice;
}

/* Counts the tokens of every expert, gives each expert whole blocks of 128 rows, and every choice its row. One CTA. */
constexpr int kMpThreads = 1024;
__global__ void __launch_bounds__(kMpThreads) lm_moe_plan_kernel(const LmMoe a, int choices, int max_blocks) {
    __shared__ int count[kLmMoeExperts], start[kLmMoeExperts], scan[2][kMpThreads];
    pdl_launch_dependents();
    pdl_wait();
    const int tid = threadIdx.x;
    for (int e = tid; e < a.experts; e += kMpThreads) count[e] = 0;
    __syncthreads();
    for (int i = tid; i < choices; i += kMpThreads) atomicAdd(&count[a.chosen[i]], 1);
    __syncthreads();
    const int mine = tid < a.experts ? (count[tid] + 127) / 128 : 0;
    int cur = 0;
    scan[0][tid] = mine;
    __syncthreads();
    for (int o = 1; o < kMpThreads; o <<= 1) {                  /* blocks up to and including this expert's */
        scan[cur ^ 1][tid] = scan[cur][tid] + (tid >= o ? scan[cur][tid - o] : 0);
        cur ^= 1;
        __syncthreads();
    }
    const int end = scan[cur][tid], first = end - mine, used = scan[cur][kMpThreads - 1];
    if (tid < a.experts) {
        for (int b = 0; b < mine; b++) {
            const int left = count[tid] - b * 128;
            if (first + b < max_blocks) a.table[first + b] = make_int4(tid, (first + b) * 128, left < 128 ? left : 128, 0);
        }
        start[tid] = first * 128;
    }
    for (int b = used + tid; b < max_blocks; b += kMpThreads) a.table[b] = make_int4(-1, 0, 0, 0);
    __syncthreads();
    for (int i = tid; i < choices; i += kMpThreads) a.at[i] = atomicAdd(&start[a.chosen[i]], 1);
}

/* Rows of the experts' input in sorted order. grid = (choices) */
__global__ void __launch_bounds__(128) lm_moe_gather_kernel(const LmMoe a, const LmSink to) {
    pdl_launch_dependents();
    pdl_wait();
    const int i = blockIdx.x, m = i / a.top, r = a.at[i];
    if (to.rows) {
        for (int c = threadIdx.x * 4; c < to.ld; c += 512)
            *reinterpret_cast<float4 *>(to.rows + (size_t)r * to.ld + c) = vb_ldcg4(a.x.rows + (size_t)m * a.x.ld + c);
    } else {
        for (int t = 0; t < to.n_terms; t++)
            for (int c = threadIdx.x * 8; c < to.ld; c += 1024)
                *reinterpret_cast<uint4 *>(to.terms + ((size_t)t * to.rows_pad + r) * to.ld + c) =
                    __ldcg(reinterpret_cast<const uint4 *>(a.x.terms + ((size_t)t * a.x.rows_pad + m) * a.x.ld + c));
    }
}

template <bool DOWN> int launch_few(const LmMoe &a, int M, cudaStream_t st) {
    static size_t set = 48 * 1024;
    const size_t smem = sizeof(float) * (DOWN ? a.down.Kp : a.up.Kp);
    if (smem > 200 * 1024) return -1;
    if (smem > set) {
        if (cudaFuncSetAttribute(lm_moe_few_kernel<DOWN>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) {
            cudaGetLastError();
            return -1;
        }
        set = smem;
    }
    const int N = DOWN ? a.width : a.ff;
    return ok(launch_pdl(lm_moe_few_kernel<DOWN>, dim3((N + kMfRows - 1) / kMfRows, M * a.top), dim3(kMfThreads), smem, st, a));
}

} // namespace

int lm_moe_blocks(int rows, int experts, int top) {
    const long long choices = (long long)rows * top;
    return (int)(choices / 128 + (choices < experts ? choices : experts));
}

int lm_moe_few(const LmMoe &a, int M, cudaStream_t st) { return launch_few<false>(a, M, st) || launch_few<true>(a, M, st) ? -1 : 0; }

int lm_moe_plan(const LmMoe &a, int M, cudaStream_t st) {
    if (a.experts > kLmMoeExperts) return -1;
    return ok(launch_pdl(lm_moe_plan_kernel, dim3(1), dim3(kMpThreads), 0, st, a, M * a.top, lm_moe_blocks(M, a.experts, a.top)));
}

int lm_moe_gather(const LmMoe &a, const LmSink &to, int M, cudaStream_t st) {
    return ok(launch_pdl(lm_moe_gather_kernel, dim3(M * a.top), dim3(128), 0, st, a, to));
}

} // namespace vb
