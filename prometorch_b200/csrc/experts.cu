// A mixture of experts for inference, the parts that take any size:
//   route_kernel        a warp per token: scores (sigmoid, or softmax over all outputs), the `top` outputs with the largest corrected scores,
//                       their weights, and the token's rank among an expert's rows (counted in shared memory, then once per CTA and expert
//                       in global memory);
//   place_kernel        prefix sums of the counts: the place of every (token, expert) pair in the order by expert, and back;
//   route_small_kernel  both for few tokens in one CTA;
//   route_rows_kernel   the router's product as well, for few tokens;
//   expert_simt_kernel  a grouped product over the sorted rows with FMAs in fp32 (fp32 models, sizes the tensor-core kernel cannot address).
// The router may have more outputs than there are experts: those behind them are identities, without rows; their place is -1.  `always` more
// experts follow the routed ones in the order of rows; every token uses them, with the weight 1.
// Where a row lies inside its expert depends on the order of atomics; what is computed for it does not.
#include "common.cuh"
#include <algorithm>

namespace ptb {
namespace moe {

constexpr int RT_WARPS = 8, RS_WARPS = 32, SMALL_TOKENS = 64;

struct Route {
    const float* z;                    // [splits][n] rows of pitch ld
    int splits;
    long long stride, ld;
    const float* correction;           // [O]
    int n, E, top;
    int O, softmax, always;            // router outputs: the experts and the identities behind them
    float scale;                       // weights: scores over their sum times scale; softmax: the scores times scale
    int* index;                        // [n][K] out: place in the order by expert, K = top + always
    float* weight;                     // [n][K] out
    int* token;                        // [n K] out
    int* offsets;                      // [E + always + 1] out
    int* expert;                       // [n][K] between the kernels, the first `top` of a row
    int* rank;                         // [n][K] likewise
    int* counts;                       // [E], zero at the start
    int* status;
    __host__ __device__ int K() const { return top + always; }
};

// Pair p of a token goes to its place; off: first place of every expert.
__device__ __forceinline__ void put(const Route& R, long long p, const int* off) {
    const int K = R.K(), i = (int)(p / K), k = (int)(p % K);
    int at;
    if (k >= R.top) at = off[R.E + k - R.top] + i;
    else {
        const int e = __ldcg(R.expert + p);
        at = e < R.E ? off[e] + R.rank[p] : -1;
    }
    R.index[p] = at;
    if (at >= 0) R.token[at] = i;
}

// The logit of token i and expert e.
struct Logits {
    const Route& R;
    int i;
    __device__ __forceinline__ float operator()(int e) const {
        float z = 0.f;
        for (int s = 0; s < R.splits; ++s) z += R.z[s * R.stride + (size_t)i * R.ld + e];
        return z;
    }
};

// One warp: choice scores of token i into c_s [O] and plain ones behind them, its `top` outputs one after the other to lane 0 of the callback.
template <typename Z, typename F>
__device__ __forceinline__ void choose(const Route& R, int i, float* c_s, Z logit, F chosen) {
    const int lane = threadIdx.x & 31;
    float* s_s = c_s + R.O;
    if (R.softmax) {
        float most = -INFINITY, all = 0.f;
        for (int e = lane; e < R.O; e += 32) {
            s_s[e] = logit(e);
            most = fmaxf(most, s_s[e]);
        }
        most = warp_max(most);
        for (int e = lane; e < R.O; e += 32) all += s_s[e] = expf(s_s[e] - most);
        all = 1.f / warp_sum(all);
        for (int e = lane; e < R.O; e += 32) {
            s_s[e] *= all;
            c_s[e] = s_s[e] + R.correction[e];
        }
    } else
        for (int e = lane; e < R.O; e += 32) {
            const float s = sigmoid(logit(e));
            s_s[e] = s;
            c_s[e] = s + R.correction[e];
        }
    __syncwarp();
    float sum = 0.f, mine = 0.f;                       // lane k keeps the score of the k-th expert (and of k + 32, ... in turn)
    for (int k = 0; k < R.top; ++k) {
        float best = -INFINITY;
        int at = R.O;
        for (int e = lane; e < R.O; e += 32)
            if (c_s[e] > best) { best = c_s[e]; at = e; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float b = __shfl_xor_sync(0xffffffffu, best, o);
            const int a = __shfl_xor_sync(0xffffffffu, at, o);
            if (b > best || (b == best && a < at)) { best = b; at = a; }
        }
        if (at >= R.O) at = k;                         // scores that are not numbers: any expert will do
        const float score = s_s[at];
        sum += score;
        if (lane == (k & 31)) mine = score;
        __syncwarp();
        if (lane == 0) {
            c_s[at] = -INFINITY;
            chosen(k, at);
        }
        __syncwarp();
        if ((k & 31) == 31 && k + 1 < R.top) R.weight[(size_t)i * R.K() + k - 31 + lane] = mine;      // unscaled: the sum is not known yet
    }
    const float f = R.softmax ? R.scale : R.scale / (sum + 1e-20f);
    const int k0 = (R.top - 1) & ~31;                  // the last ones are still in registers
    for (int k = lane; k < k0; k += 32) R.weight[(size_t)i * R.K() + k] *= f;
    if (k0 + lane < R.top) R.weight[(size_t)i * R.K() + k0 + lane] = mine * f;
    for (int k = R.top + lane; k < R.K(); k += 32) R.weight[(size_t)i * R.K() + k] = 1.f;
}

__global__ void __launch_bounds__(RT_WARPS * 32) route_kernel(const __grid_constant__ Route R) {
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5;
    float* c_s = smem + warp * 2 * R.O;
    int* count = reinterpret_cast<int*>(smem + RT_WARPS * 2 * R.O);
    int* base = count + R.E;
    for (int e = threadIdx.x; e < R.E; e += blockDim.x) count[e] = 0;
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    const int i = blockIdx.x * RT_WARPS + warp;
    if (i < R.n)
        choose(R, i, c_s, Logits{R, i}, [&](int k, int e) {
            R.expert[(size_t)i * R.K() + k] = e;
            if (e < R.E) R.rank[(size_t)i * R.K() + k] = atomicAdd(&count[e], 1);
        });
    __syncthreads();
    for (int e = threadIdx.x; e < R.E; e += blockDim.x) base[e] = count[e] ? atomicAdd(&R.counts[e], count[e]) : 0;
    __syncthreads();
    if (i < R.n)
        for (int k = threadIdx.x & 31; k < R.top; k += 32) {
            const size_t p = (size_t)i * R.K() + k;
            if (R.expert[p] < R.E) R.rank[p] += base[R.expert[p]];
        }
}

// Exclusive sums of the experts' rows to off[0 .. E + always], by the first warp; count: of the routed ones.
__device__ __forceinline__ void prefix(const Route& R, const int* count, int* off) {
    if (threadIdx.x < 32) {
        const int E = R.E + R.always;
        int run = 0;
        for (int e0 = 0; e0 < E; e0 += 32) {
            const int e = e0 + threadIdx.x, v = e < R.E ? count[e] : e < E ? R.n : 0;
            int s = v;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int t = __shfl_up_sync(0xffffffffu, s, o);
                if ((int)threadIdx.x >= o) s += t;
            }
            if (e < E) off[e] = run + s - v;
            run += __shfl_sync(0xffffffffu, s, 31);
        }
        if (threadIdx.x == 0) off[E] = run;
    }
}

__global__ void __launch_bounds__(256) place_kernel(const __grid_constant__ Route R) {
    extern __shared__ int off[];
    pdl_wait();
    pdl_launch_dependents();
    prefix(R, R.counts, off);
    __syncthreads();
    if (blockIdx.x == 0)
        for (int e = threadIdx.x; e <= R.E + R.always; e += blockDim.x) R.offsets[e] = off[e];
    const long long total = (long long)R.n * R.K();
    for (long long p = (long long)blockIdx.x * blockDim.x + threadIdx.x; p < total; p += (long long)gridDim.x * blockDim.x) put(R, p, off);
}

__global__ void __launch_bounds__(RS_WARPS * 32) route_small_kernel(const __grid_constant__ Route R) {
    extern __shared__ float smem[];
    const int warp = threadIdx.x >> 5;
    float* c_s = smem + warp * 2 * R.O;
    int* count = reinterpret_cast<int*>(smem + RS_WARPS * 2 * R.O);
    int* off = count + R.E;
    for (int e = threadIdx.x; e < R.E; e += blockDim.x) count[e] = 0;
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    for (int i = warp; i < R.n; i += RS_WARPS)
        choose(R, i, c_s, Logits{R, i}, [&](int k, int e) {
            R.expert[(size_t)i * R.K() + k] = e;
            if (e < R.E) R.rank[(size_t)i * R.K() + k] = atomicAdd(&count[e], 1);
        });
    __syncthreads();
    prefix(R, count, off);
    __syncthreads();
    for (int e = threadIdx.x; e <= R.E + R.always; e += blockDim.x) R.offsets[e] = off[e];
    for (int p = threadIdx.x; p < R.n * R.K(); p += blockDim.x) put(R, p, off);
}

constexpr int RR_THREADS = 128, RR_WARPS = RR_THREADS / 32;

// CTA (x, token): every gridDim.x-th group of RR_WARPS experts, a warp per expert.  Of a token's CTAs the last one to finish chooses; of the
// tokens the last one puts all pairs in order.  h [n][W] of pitch ldh, w [O][W], both bf16 or fp32; z [n][O].  done [n + 1]: zero before
// and after.
template <typename T>
__global__ void __launch_bounds__(RR_THREADS) route_rows_kernel(const __grid_constant__ Route R, const T* __restrict__ h, long long ldh, const T* __restrict__ w, int W,
                                                                float* z, unsigned* done) {
    extern __shared__ float c_s[];                     // [2 O], later counts [E] and offsets [E + always + 1]
    __shared__ int last;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, i = blockIdx.y;
    constexpr int V = 16 / sizeof(T);                  // elements of a 16-byte load
    const bool vec = W % V == 0 && ldh % V == 0 && (((uintptr_t)w | (uintptr_t)h) & 15) == 0;
    pdl_wait();
    pdl_launch_dependents();
    const T* x = h + (size_t)i * ldh;
    for (int e = blockIdx.x * RR_WARPS + warp; e < R.O; e += gridDim.x * RR_WARPS) {
        const T* row = w + (size_t)e * W;
        float a = 0.f;
        if (vec) {
#pragma unroll 8
            for (int c = lane * V; c < W; c += 32 * V) {
                const uint4 p = *reinterpret_cast<const uint4*>(row + c), q = *reinterpret_cast<const uint4*>(x + c);
                const T* u = reinterpret_cast<const T*>(&p);
                const T* v = reinterpret_cast<const T*>(&q);
#pragma unroll
                for (int k = 0; k < V; ++k) a = fmaf((float)u[k], (float)v[k], a);
            }
        } else
            for (int c = lane; c < W; c += 32) a = fmaf((float)row[c], (float)x[c], a);
        a = warp_sum(a);
        if (lane == 0) z[(size_t)i * R.O + e] = a;
    }
    auto finished = [&](unsigned* counter, unsigned of) {          // whether this CTA is the last of `of` to come here
        __threadfence();
        __syncthreads();
        if (threadIdx.x == 0) {
            last = atomicAdd(counter, 1u) == of - 1;
            if (last) *counter = 0;
        }
        __syncthreads();
        if (last) __threadfence();
        return last != 0;
    };
    if (!finished(done + i, gridDim.x)) return;
    if (warp == 0) choose(R, i, c_s, [&](int e) { return __ldcg(z + (size_t)i * R.O + e); }, [&](int k, int e) { R.expert[(size_t)i * R.K() + k] = e; });
    if (!finished(done + R.n, gridDim.y)) return;
    int *count = reinterpret_cast<int*>(c_s), *off = count + R.E;
    for (int e = threadIdx.x; e < R.E; e += RR_THREADS) count[e] = 0;
    __syncthreads();
    const int K = R.K(), pairs = R.n * K;
    for (int p = threadIdx.x; p < pairs; p += RR_THREADS) {
        if (p % K >= R.top) continue;
        const int e = __ldcg(R.expert + p);
        if (e < R.E) R.rank[p] = atomicAdd(&count[e], 1);
    }
    __syncthreads();
    prefix(R, count, off);
    __syncthreads();
    for (int e = threadIdx.x; e <= R.E + R.always; e += RR_THREADS) R.offsets[e] = off[e];
    for (int p = threadIdx.x; p < pairs; p += RR_THREADS) put(R, p, off);
}

// ---------------------------------------------------------------------------------------------- grouped product, any size
constexpr int ST_M = 32, ST_N = 64, ST_K = 32;

template <typename T> __device__ __forceinline__ float f32_of(T v) { return (float)v; }

// 32 sorted rows of one expert x 64 output columns per CTA; GATED: B has gate rows [0, N) and up rows [N, 2 N).
template <typename T, bool GATED>
__global__ void __launch_bounds__(256) expert_simt_kernel(const T* __restrict__ a, const int* __restrict__ token, long long lda, const T* __restrict__ b,
                                                          T* __restrict__ out, const int* __restrict__ offsets, int rows, int E, int N, int K) {
    __shared__ float as[ST_K][ST_M + 1], gs[ST_K][ST_N + 1], us[GATED ? ST_K : 1][ST_N + 1];
    __shared__ int where[3];
    pdl_wait();
    pdl_launch_dependents();
    if (threadIdx.x == 0) {                            // the expert and the rows of tile blockIdx.y
        int t = blockIdx.y;
        where[0] = -1;
        for (int e = 0; e < E; ++e) {
            const int lo = offsets[e], hi = offsets[e + 1], tiles = (hi - lo + ST_M - 1) / ST_M;
            if (t < tiles) { where[0] = e; where[1] = lo + t * ST_M; where[2] = min(hi, lo + (t + 1) * ST_M); break; }
            t -= tiles;
        }
    }
    __syncthreads();
    const int e = where[0], r0 = where[1], r1 = min(where[2], rows), n0 = blockIdx.x * ST_N;
    if (e < 0) return;
    const T* be = b + (size_t)e * (GATED ? 2 : 1) * N * K;
    const int tx = threadIdx.x & 31, ty = threadIdx.x >> 5;            // columns tx, tx + 32; rows ty + 8 i
    float g[4][2], u[4][2];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) g[i][j] = u[i][j] = 0.f;
    for (int k0 = 0; k0 < K; k0 += ST_K) {
        for (int i = threadIdx.x; i < ST_M * ST_K; i += 256) {
            const int r = i / ST_K, k = k0 + i % ST_K;
            float v = 0.f;
            if (r0 + r < r1 && k < K) v = f32_of<T>(a[(size_t)(token ? token[r0 + r] : r0 + r) * lda + k]);
            as[i % ST_K][r] = v;
        }
        for (int i = threadIdx.x; i < ST_N * ST_K; i += 256) {
            const int n = n0 + i / ST_K, k = k0 + i % ST_K;
            const bool in = n < N && k < K;
            gs[i % ST_K][i / ST_K] = in ? f32_of<T>(be[(size_t)n * K + k]) : 0.f;
            if constexpr (GATED) us[i % ST_K][i / ST_K] = in ? f32_of<T>(be[(size_t)(N + n) * K + k]) : 0.f;
        }
        __syncthreads();
#pragma unroll 8
        for (int k = 0; k < ST_K; ++k)
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float x = as[k][ty + 8 * i];
#pragma unroll
                for (int j = 0; j < 2; ++j) {
                    g[i][j] = fmaf(x, gs[k][tx + 32 * j], g[i][j]);
                    if constexpr (GATED) u[i][j] = fmaf(x, us[k][tx + 32 * j], u[i][j]);
                }
            }
        __syncthreads();
    }
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int r = r0 + ty + 8 * i, n = n0 + tx + 32 * j;
            if (r < r1 && n < N) out[(size_t)r * N + n] = (T)(GATED ? silu(g[i][j]) * u[i][j] : g[i][j]);
        }
}

}  // namespace moe
}  // namespace ptb

using namespace ptb;

// Routing of n tokens over O >= E router outputs: z [splits][n] fp32 logits (rows of pitch ld, splits `stride` apart), correction [O].  `always`
// experts behind the E routed ones serve every token; K = top + always.  index [n, K]: the place of a token's i-th expert in the order by expert, -1
// for an output behind the routed experts; weight [n, K]: its sigmoid score over the sum of the chosen ones, times scale (softmax: its score times
// scale), 1 for the last `always`; token [n K]: the token of every place; offsets [E + always + 1].  work: 2 n K + E ints.
PTB_API int ptb_expert_route(const float* z, int splits, long long stride, long long ld, const float* correction, int n, int E, int O, int always, int softmax, int top, float scale,
                             int* index, float* weight, int* token, int* offsets, int* work, int* status, cudaStream_t st) {
    using namespace ptb::moe;
    if (n <= 0) return 0;
    if (E < 1 || O < E || top < 1 || top > O || O > 1024 || always < 0 || E + always > 1024) {
        ptb_set_error("experts: %d of %d outputs (at most 1024), %d and %d experts", top, O, E, always);
        return -1;
    }
    const size_t pairs = (size_t)n * (top + always);
    Route r{z, splits, stride, ld, correction, n, E, top, O, softmax, always, scale, index, weight, token, offsets, work, work + pairs, work + 2 * pairs, status};
    const bool pdl = ptb_pdl_enabled();
    if (n <= SMALL_TOKENS && O <= 256) {
        const size_t smem = ((size_t)RS_WARPS * 2 * O + 2 * E + always + 1) * 4;
        if (smem > 48 * 1024) PTB_CUDA_OK(cudaFuncSetAttribute(route_small_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
        PTB_CUDA_OK(ptb_launch(route_small_kernel, dim3(1), dim3(RS_WARPS * 32), smem, st, pdl, r));
    } else {
        PTB_CUDA_OK(cudaMemsetAsync(r.counts, 0, (size_t)E * 4, st));
        const size_t smem = ((size_t)RT_WARPS * 2 * O + 2 * E) * 4;
        if (smem > 48 * 1024) PTB_CUDA_OK(cudaFuncSetAttribute(route_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024));
        PTB_CUDA_OK(ptb_launch(route_kernel, dim3((n + RT_WARPS - 1) / RT_WARPS), dim3(RT_WARPS * 32), smem, st, false, r));
        PTB_CUDA_OK(ptb_launch(place_kernel, dim3((unsigned)std::min<size_t>(1024, (pairs + 255) / 256)), dim3(256), (size_t)(E + always + 1) * 4, st, pdl, r));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// The same from the rows themselves, for few tokens: h [n, W] (pitch ldh) and the router w [O, W], both bf16 or fp32.  work: 2 n K ints and n O floats;
// done: n + 1 unsigned that are zero between calls, used by one stream at a time.
PTB_API int ptb_expert_route_rows(const void* h, long long ldh, const void* w, int W, const float* correction, int n, int E, int O, int always, int softmax, int top,
                                  float scale, int* index, float* weight, int* token, int* offsets, int* work, unsigned* done, int bf16, cudaStream_t st) {
    using namespace ptb::moe;
    if (n <= 0) return 0;
    const size_t pairs = (size_t)n * (top + always);
    if (E < 1 || O < E || top < 1 || top > O || O > 1024 || always < 0 || E + always > 1024 || n > 65535 || W < 1) {
        ptb_set_error("experts: %d of %d outputs (at most 1024), %d and %d experts, %d columns", top, O, E, always, W);
        return -1;
    }
    const Route r{nullptr, 0, 0, 0, correction, n, E, top, O, softmax, always, scale, index, weight, token, offsets, work, work + pairs, nullptr, nullptr};
    const bool pdl = ptb_pdl_enabled();
    auto go = [&](auto k, auto t) {
        using T = decltype(t);
        const int groups = std::max(1, std::min((O + RR_WARPS - 1) / RR_WARPS, 148 * 8 / n));
        return ptb_launch(k, dim3(groups, n), dim3(RR_THREADS), (2 * (size_t)O + always + 1) * 4, st, pdl, r, (const T*)h, ldh, (const T*)w, W,
                          reinterpret_cast<float*>(work + 2 * pairs), done);
    };
    PTB_CUDA_OK(bf16 ? go(route_rows_kernel<__nv_bfloat16>, __nv_bfloat16()) : go(route_rows_kernel<float>, 0.f));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out [rows, N] = A_e B_e^T for the rows of every expert e (offsets [E + 1]), in fp32 arithmetic; `gated`: B_e has 2 N rows and the result is
// silu(gate) * up.  Row r of A is a[token[r]] (token null: a[r]), pitch lda.  bf16 or fp32 operands and result.
PTB_API int ptb_expert_gemm_simt(const void* a, const int* token, long long lda, const void* b, int gated, void* out, const int* offsets, int rows, int E, int N,
                                 int K, int bf16, int* status, cudaStream_t st) {
    using namespace ptb::moe;
    (void)status;
    if (rows <= 0 || N <= 0 || K <= 0) return 0;
    const long long tiles = std::min<long long>((long long)rows, rows / ST_M + E);
    if (tiles > 65535) { ptb_set_error("experts: %d rows in one launch", rows); return -1; }
    const dim3 grid((N + ST_N - 1) / ST_N, (unsigned)tiles);
    const bool pdl = ptb_pdl_enabled();
    auto go = [&](auto k, auto t) {
        using T = decltype(t);
        return ptb_launch(k, grid, dim3(256), 0, st, pdl, (const T*)a, token, lda, (const T*)b, (T*)out, offsets, rows, E, N, K);
    };
    if (bf16) PTB_CUDA_OK(gated ? go(expert_simt_kernel<__nv_bfloat16, true>, __nv_bfloat16()) : go(expert_simt_kernel<__nv_bfloat16, false>, __nv_bfloat16()));
    else PTB_CUDA_OK(gated ? go(expert_simt_kernel<float, true>, 0.f) : go(expert_simt_kernel<float, false>, 0.f));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
