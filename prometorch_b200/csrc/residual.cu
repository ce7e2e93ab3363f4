// Kernels around an fp32 residual stream, for decoders that keep the sum of their sublayers in 32-bit while the matrix
// products run on bf16 copies:
//   embed_residual_kernel   x = table[id] * scale (fp32) and its copy in the compute type;
//   post_norm_add_kernel    x += rmsnorm(y) * g: the norm sits on a sublayer's output, before the sum;
//   row_norm_kernel         rmsnorm of chosen rows of x, in the compute type (the model's last norm).
// A norm's weight is a vector, a single number, or both.  T is the compute type (bf16 or float); with float the copy is x itself
// and the `xb` pointers are null.
#include "common.cuh"
#include <algorithm>

namespace ptb {

constexpr int RS_THREADS = 256;
constexpr int RS_KEEP = 8;             // 4-element chunks a thread keeps in registers; wider rows are read again

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 raw = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
    return make_float4(a.x, a.y, b.x, b.y);
}
__device__ __forceinline__ void store4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void store4(__nv_bfloat16* p, float4 v) {
    __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<uint32_t*>(&a), *reinterpret_cast<uint32_t*>(&b));
}
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ float to_f(__nv_bfloat16 v) { return __bfloat162float(v); }
__device__ __forceinline__ void from_f(float* p, float v) { *p = v; }
__device__ __forceinline__ void from_f(__nv_bfloat16* p, float v) { *p = __float2bfloat16_rn(v); }

// Sum over the CTA, returned to every thread.
__device__ __forceinline__ float cta_sum(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    float t = (threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f;
    return warp_sum(t);
}

template <typename T>
__global__ void __launch_bounds__(RS_THREADS) embed_residual_kernel(const int* __restrict__ ids, int id_stride, const T* __restrict__ table,
                                                                    int V, int W, float scale, float* __restrict__ x, T* __restrict__ xb,
                                                                    int* status) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t row = blockIdx.x;
    int id = ids[row * id_stride];
    if (id < 0 || id >= V) {
        if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
        id = 0;
    }
    const T* src = table + (size_t)id * W;
    for (int c = threadIdx.x; c < W; c += RS_THREADS) {
        const float v = to_f(src[c]) * scale;
        x[row * W + c] = v;
        if (xb) from_f(xb + row * W + c, v);
    }
}

template <typename T, bool VEC>
__global__ void __launch_bounds__(RS_THREADS) post_norm_add_kernel(const T* __restrict__ y, long long ldy, const float* __restrict__ w, float g,
                                                                   float eps, float* __restrict__ x, T* __restrict__ xb, int W) {
    __shared__ float red[32];
    pdl_wait();
    pdl_launch_dependents();
    const size_t row = blockIdx.x;
    const T* yr = y + row * ldy;
    float* xr = x + row * W;
    float ss = 0.f;
    if constexpr (VEC) {
        const int nc = W / 4;
        float4 keep[RS_KEEP];
#pragma unroll
        for (int k = 0; k < RS_KEEP; ++k) {
            const int c = k * RS_THREADS + threadIdx.x;
            if (c < nc) {
                const float4 v = keep[k] = load4<T>(yr + (size_t)c * 4);
                ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
            }
        }
        for (int c = RS_KEEP * RS_THREADS + threadIdx.x; c < nc; c += RS_THREADS) {
            const float4 v = load4<T>(yr + (size_t)c * 4);
            ss += v.x * v.x + v.y * v.y + v.z * v.z + v.w * v.w;
        }
        const float rs = rsqrtf(cta_sum(ss, red) / (float)W + eps) * g;
        auto put = [&](int c, float4 v) {
            float4 r = *reinterpret_cast<const float4*>(xr + (size_t)c * 4);
            float4 m = make_float4(1.f, 1.f, 1.f, 1.f);
            if (w) m = *reinterpret_cast<const float4*>(w + (size_t)c * 4);
            r.x += v.x * rs * m.x; r.y += v.y * rs * m.y; r.z += v.z * rs * m.z; r.w += v.w * rs * m.w;
            store4(xr + (size_t)c * 4, r);
            if (xb) store4(xb + row * W + (size_t)c * 4, r);
        };
#pragma unroll
        for (int k = 0; k < RS_KEEP; ++k) {
            const int c = k * RS_THREADS + threadIdx.x;
            if (c < nc) put(c, keep[k]);
        }
        for (int c = RS_KEEP * RS_THREADS + threadIdx.x; c < nc; c += RS_THREADS) put(c, load4<T>(yr + (size_t)c * 4));
    } else {
        for (int c = threadIdx.x; c < W; c += RS_THREADS) { const float v = to_f(yr[c]); ss += v * v; }
        const float rs = rsqrtf(cta_sum(ss, red) / (float)W + eps) * g;
        for (int c = threadIdx.x; c < W; c += RS_THREADS) {
            const float r = xr[c] + to_f(yr[c]) * rs * (w ? w[c] : 1.f);
            xr[c] = r;
            if (xb) from_f(xb + row * W + c, r);
        }
    }
}

template <typename T>
__global__ void __launch_bounds__(RS_THREADS) row_norm_kernel(const float* __restrict__ x, const long long* __restrict__ index, int rows,
                                                              const float* __restrict__ w, float g, float eps, T* __restrict__ out, int W,
                                                              int* status) {
    __shared__ float red[32];
    pdl_wait();
    pdl_launch_dependents();
    const size_t o = blockIdx.x;
    long long r = index ? index[o] : (long long)o;
    if (r < 0 || r >= rows) {
        if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
        r = 0;
    }
    const float* xr = x + (size_t)r * W;
    float ss = 0.f;
    for (int c = threadIdx.x; c < W; c += RS_THREADS) ss += xr[c] * xr[c];
    const float rs = rsqrtf(cta_sum(ss, red) / (float)W + eps) * g;
    for (int c = threadIdx.x; c < W; c += RS_THREADS) from_f(out + o * W + c, xr[c] * rs * (w ? w[c] : 1.f));
}

}  // namespace ptb

using namespace ptb;

// x [n, W] fp32 = table[ids[i * id_stride]] * scale; xb: its bf16 copy (bf16 != 0; the table has the same type).
PTB_API int ptb_embed_residual(const int* ids, int id_stride, const void* table, int V, int W, float scale, int n, float* x, void* xb,
                               int* status, int bf16, cudaStream_t st) {
    if (n <= 0) return 0;
    const bool pdl = ptb_pdl_enabled();
    if (bf16)
        PTB_CUDA_OK(ptb_launch(embed_residual_kernel<__nv_bfloat16>, dim3(n), dim3(RS_THREADS), 0, st, pdl, ids, id_stride, (const __nv_bfloat16*)table, V, W,
                               scale, x, (__nv_bfloat16*)xb, status));
    else
        PTB_CUDA_OK(ptb_launch(embed_residual_kernel<float>, dim3(n), dim3(RS_THREADS), 0, st, pdl, ids, id_stride, (const float*)table, V, W, scale, x,
                               (float*)nullptr, status));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// x [n, W] fp32 += y / rms(y) * g * w, with y [n, W] (row pitch ldy) in bf16 or fp32; xb: the bf16 copy of the new x.  w: optional
// fp32 [W].  eps sits inside the root.
PTB_API int ptb_post_norm_add(const void* y, long long ldy, const float* w, float g, float eps, float* x, void* xb, int n, int W, int bf16,
                              cudaStream_t st) {
    if (n <= 0) return 0;
    const bool pdl = ptb_pdl_enabled();
    const bool vec = W % 4 == 0 && ldy % 4 == 0 && (((uintptr_t)y | (uintptr_t)x | (uintptr_t)xb | (uintptr_t)w) & 15) == 0;
    if (bf16) {
        auto k = vec ? post_norm_add_kernel<__nv_bfloat16, true> : post_norm_add_kernel<__nv_bfloat16, false>;
        PTB_CUDA_OK(ptb_launch(k, dim3(n), dim3(RS_THREADS), 0, st, pdl, (const __nv_bfloat16*)y, ldy, w, g, eps, x, (__nv_bfloat16*)xb, W));
    } else {
        auto k = vec ? post_norm_add_kernel<float, true> : post_norm_add_kernel<float, false>;
        PTB_CUDA_OK(ptb_launch(k, dim3(n), dim3(RS_THREADS), 0, st, pdl, (const float*)y, ldy, w, g, eps, x, (float*)nullptr, W));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out [m, W] (bf16 or fp32) = x[index[i]] / rms * g * w for m rows of x [rows, W] fp32; index null: the first m rows.
PTB_API int ptb_row_norm(const float* x, const long long* index, int rows, const float* w, float g, float eps, void* out, int m, int W,
                         int* status, int bf16, cudaStream_t st) {
    if (m <= 0) return 0;
    const bool pdl = ptb_pdl_enabled();
    if (bf16)
        PTB_CUDA_OK(ptb_launch(row_norm_kernel<__nv_bfloat16>, dim3(m), dim3(RS_THREADS), 0, st, pdl, x, index, rows, w, g, eps, (__nv_bfloat16*)out, W, status));
    else
        PTB_CUDA_OK(ptb_launch(row_norm_kernel<float>, dim3(m), dim3(RS_THREADS), 0, st, pdl, x, index, rows, w, g, eps, (float*)out, W, status));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
