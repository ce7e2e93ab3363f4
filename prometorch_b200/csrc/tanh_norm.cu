// Elementwise norms y = tanh(alpha x) w + b (dynamic tanh) around an fp32 residual stream:
//   tanh_residual_kernel   x += post(y); x += table[id]; out = pre(x).  y is a product in bf16 or fp32, a sum of split-K partials, or the
//                          weighed sum of the rows that a token's experts left;
//   tanh_rows_kernel       the norm of chosen rows of x;
//   softcap_kernel         cap tanh(z / cap) of logits.
// Nothing depends on a row as a whole: a thread keeps the weights of its columns in registers and walks the rows.
#include "common.cuh"
#include "ptb200_types.h"
#include <algorithm>

namespace ptb {

constexpr int TN_THREADS = 256;

template <int V> struct Vals { float v[V]; };
template <int V, typename T>
__device__ __forceinline__ Vals<V> ld(const T* p) {
    Vals<V> r;
    if constexpr (V == 4 && sizeof(T) == 4) {
        const float4 f = *reinterpret_cast<const float4*>(p);
        r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w;
    } else if constexpr (V == 4) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = (float)p[e];
    }
    return r;
}
template <int V, typename T>
__device__ __forceinline__ void st(T* p, const Vals<V>& r) {
    if constexpr (V == 4 && sizeof(T) == 4) *reinterpret_cast<float4*>(p) = make_float4(r.v[0], r.v[1], r.v[2], r.v[3]);
    else if constexpr (V == 4) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else {
#pragma unroll
        for (int e = 0; e < V; ++e) p[e] = (T)r.v[e];
    }
}

// TY: type of y, T: of out and the table.
template <typename T, typename TY, int V>
__global__ void __launch_bounds__(TN_THREADS) tanh_residual_kernel(const __grid_constant__ PtbTanhResidual P) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * V;
    const bool live = c < P.W;
    Vals<V> wo, bo, wi, bi;
    if (live) {                                        // weights of the model: no kernel before this one writes them
        wo = ld<V>(P.post_w + c);
        bo = ld<V>(P.post_b + c);
        if (P.pre_w) { wi = ld<V>(P.pre_w + c); bi = ld<V>(P.pre_b + c); }
    }
    pdl_wait();
    pdl_launch_dependents();
    if (!live) return;
    for (int row = blockIdx.y; row < P.n; row += gridDim.y) {
        Vals<V> x = ld<V>(P.x + (size_t)row * P.W + c), y;
        if (P.index) {
#pragma unroll
            for (int e = 0; e < V; ++e) y.v[e] = 0.f;
#pragma unroll 4
            for (int k = 0; k < P.top; ++k) {
                int r = P.index[(size_t)row * P.top + k];
                const float f = P.weight[(size_t)row * P.top + k];
                if (r < 0 || r >= P.y_rows) {
                    if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
                    r = 0;
                }
                const Vals<V> t = ld<V>((const TY*)P.y + (size_t)r * P.ld + c);
#pragma unroll
                for (int e = 0; e < V; ++e) y.v[e] = fmaf(f, t.v[e], y.v[e]);
            }
        } else {
            const TY* p = (const TY*)P.y + (size_t)row * P.ld + c;
            y = ld<V>(p);
#pragma unroll 4
            for (int s = 1; s < P.splits; ++s) {
                const Vals<V> t = ld<V>(p + s * P.stride);
#pragma unroll
                for (int e = 0; e < V; ++e) y.v[e] += t.v[e];
            }
        }
#pragma unroll
        for (int e = 0; e < V; ++e) x.v[e] += fmaf(tanh_accurate(P.post_alpha * y.v[e]), wo.v[e], bo.v[e]);
        if (P.ids) {
            int id = P.ids[(size_t)row * P.id_stride];
            if (id < 0 || id >= P.V) {
                if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
                id = 0;
            }
            const Vals<V> t = ld<V>((const T*)P.table + (size_t)id * P.W + c);
#pragma unroll
            for (int e = 0; e < V; ++e) x.v[e] += t.v[e];
        }
        st<V>(P.x + (size_t)row * P.W + c, x);
        if (P.pre_w) {
#pragma unroll
            for (int e = 0; e < V; ++e) x.v[e] = fmaf(tanh_accurate(P.pre_alpha * x.v[e]), wi.v[e], bi.v[e]);
            st<V>((T*)P.out + (size_t)row * P.W + c, x);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(TN_THREADS) tanh_rows_kernel(const float* __restrict__ x, const long long* __restrict__ index, int rows, float alpha,
                                                               const float* __restrict__ w, const float* __restrict__ b, T* __restrict__ out, int W, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t o = blockIdx.x;
    long long r = index ? index[o] : (long long)o;
    if (r < 0 || r >= rows) {
        if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
        r = 0;
    }
    for (int c = threadIdx.x; c < W; c += TN_THREADS) out[o * W + c] = (T)fmaf(tanh_accurate(alpha * x[(size_t)r * W + c]), w[c], b[c]);
}

__global__ void __launch_bounds__(TN_THREADS) softcap_kernel(const float* __restrict__ z, float* __restrict__ out, int V, long long ld, float cap) {
    pdl_wait();
    pdl_launch_dependents();
    const int c = blockIdx.x * TN_THREADS + threadIdx.x;
    if (c < V) out[(size_t)blockIdx.y * V + c] = cap * tanh_accurate(z[(size_t)blockIdx.y * ld + c] / cap);
}

template <typename T, typename TY>
static cudaError_t tanh_residual_launch(const PtbTanhResidual& p, bool vec, cudaStream_t s) {
    // few rows: small CTAs spread a row over more SMs; many: up to eight CTAs of 256 threads per SM walk them
    const bool many = p.n >= 1024;
    const int lanes = vec ? p.W / 4 : p.W, threads = std::min(many ? TN_THREADS : 64, (lanes + 31) / 32 * 32), cols = (lanes + threads - 1) / threads;
    const int rows = std::max(1, std::min(p.n, 148 * 8 * (TN_THREADS / threads) / cols));
    auto go = [&](auto k) { return ptb_launch(k, dim3(cols, std::min(rows, 65535)), dim3(threads), 0, s, ptb_pdl_enabled(), p); };
    return vec ? go(tanh_residual_kernel<T, TY, 4>) : go(tanh_residual_kernel<T, TY, 1>);
}

}  // namespace ptb

using namespace ptb;

// x [n, W] fp32 += post(y); += table[ids]; out = pre(x); see PtbTanhResidual.
PTB_API int ptb_tanh_residual(const PtbTanhResidual* args, cudaStream_t s) {
    const PtbTanhResidual& p = *args;
    if (p.n <= 0) return 0;
    if (!p.y || !p.post_w || !p.post_b || (p.pre_w && (!p.pre_b || !p.out)) || (p.splits > 1 && !p.f32) || (p.index && (!p.weight || p.top < 1)) || (p.ids && !p.table)) {
        ptb_set_error("tanh_residual: missing operand");
        return -1;
    }
    const uintptr_t bases = (uintptr_t)p.x | (uintptr_t)p.y | (uintptr_t)p.post_w | (uintptr_t)p.post_b | (uintptr_t)p.pre_w | (uintptr_t)p.pre_b | (uintptr_t)p.table |
                            (uintptr_t)p.out;
    const bool vec = p.W % 4 == 0 && p.ld % 4 == 0 && p.stride % 4 == 0 && (bases & 15) == 0;
    cudaError_t e;
    if (p.bf16) e = p.f32 ? tanh_residual_launch<__nv_bfloat16, float>(p, vec, s) : tanh_residual_launch<__nv_bfloat16, __nv_bfloat16>(p, vec, s);
    else e = p.f32 ? tanh_residual_launch<float, float>(p, vec, s) : tanh_residual_launch<float, __nv_bfloat16>(p, vec, s);
    PTB_CUDA_OK(e);
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out [m, W] (bf16 or fp32) = tanh(alpha x[index[i]]) w + b for m rows of x [rows, W] fp32; index null: the first m rows.
PTB_API int ptb_tanh_rows(const float* x, const long long* index, int rows, float alpha, const float* w, const float* b, void* out, int m, int W, int* status,
                          int bf16, cudaStream_t s) {
    if (m <= 0) return 0;
    const bool pdl = ptb_pdl_enabled();
    if (bf16) PTB_CUDA_OK(ptb_launch(tanh_rows_kernel<__nv_bfloat16>, dim3(m), dim3(TN_THREADS), 0, s, pdl, x, index, rows, alpha, w, b, (__nv_bfloat16*)out, W, status));
    else PTB_CUDA_OK(ptb_launch(tanh_rows_kernel<float>, dim3(m), dim3(TN_THREADS), 0, s, pdl, x, index, rows, alpha, w, b, (float*)out, W, status));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out [m, V] = cap tanh(z / cap), z fp32 with row pitch ld.
PTB_API int ptb_softcap(const float* z, float* out, int m, int V, long long ld, float cap, cudaStream_t s) {
    if (m <= 0 || V <= 0) return 0;
    for (int lo = 0; lo < m; lo += 65535)
        PTB_CUDA_OK(ptb_launch(softcap_kernel, dim3((V + TN_THREADS - 1) / TN_THREADS, std::min(65535, m - lo)), dim3(TN_THREADS), 0, s, ptb_pdl_enabled(),
                               z + (size_t)lo * ld, out + (size_t)lo * V, V, ld, cap));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
