// Kernels around an fp32 residual stream, for decoders that keep the sum of their sublayers in 32-bit while the matrix
// products run on bf16 copies:
//   embed_residual_kernel   x = table[id] * scale (fp32) and its copy in the compute type;
//   residual_norm_kernel    x += the sum of one or two sublayer outputs (each RMS-normed first if it has a weight; bf16, fp32 or
//                           split-K partials), then h = rmsnorm(x) * w for the next sublayer;
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

// A sublayer's output on its way into the stream: y = sum over `splits` partials (pitch ld), times g, and w / rms(y) if there is a w.
struct Branch {
    const void* y;                     // null: absent
    int f32, splits;
    long long stride, ld;
    const float* w;
    float g;
};
template <int V> struct Row { float v[V]; };
template <int V>
__device__ __forceinline__ Row<V> branch_load(const Branch& B, size_t row, int c) {
    Row<V> r;
    if (B.f32) {
        const float* p = (const float*)B.y + row * B.ld + c;
        if constexpr (V == 4) { const float4 a = load4<float>(p); r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w; }
        else r.v[0] = *p;
        for (int s = 1; s < B.splits; ++s) {
            p += B.stride;
            if constexpr (V == 4) { const float4 a = load4<float>(p); r.v[0] += a.x; r.v[1] += a.y; r.v[2] += a.z; r.v[3] += a.w; }
            else r.v[0] += *p;
        }
    } else {
        const __nv_bfloat16* p = (const __nv_bfloat16*)B.y + row * B.ld + c;
        if constexpr (V == 4) { const float4 a = load4<__nv_bfloat16>(p); r.v[0] = a.x; r.v[1] = a.y; r.v[2] = a.z; r.v[3] = a.w; }
        else r.v[0] = to_f(*p);
    }
    return r;
}

// One CTA per row.  A thread keeps NK groups of V elements of x and of both branches in registers; wider rows are read again.
template <typename T, int V, int NK, int NB>
__global__ void __launch_bounds__(RS_THREADS) residual_norm_kernel(const Branch A, const Branch B, float eps, float* __restrict__ x,
                                                                   const float* __restrict__ w, T* __restrict__ out, int W) {
    __shared__ float red[4][32];
    pdl_wait();
    pdl_launch_dependents();
    const size_t row = blockIdx.x;
    float* xr = x + row * W;
    const int nc = W / V, kept = NK * RS_THREADS;
    Row<V> a[NK], b[NB == 2 ? NK : 1], xs[NK];
    float sa = 0.f, sb = 0.f;
#pragma unroll
    for (int k = 0; k < NK; ++k) {
        const int c = k * RS_THREADS + threadIdx.x;
        if (c < nc) {
            a[k] = branch_load<V>(A, row, c * V);
            if constexpr (NB == 2) b[k] = branch_load<V>(B, row, c * V);
            if constexpr (V == 4) { const float4 t = load4<float>(xr + c * 4); xs[k].v[0] = t.x; xs[k].v[1] = t.y; xs[k].v[2] = t.z; xs[k].v[3] = t.w; }
            else xs[k].v[0] = xr[c];
#pragma unroll
            for (int e = 0; e < V; ++e) {
                sa += a[k].v[e] * a[k].v[e];
                if constexpr (NB == 2) sb += b[k].v[e] * b[k].v[e];
            }
        }
    }
    for (int c = kept + threadIdx.x; c < nc; c += RS_THREADS) {
        const Row<V> r = branch_load<V>(A, row, c * V);
#pragma unroll
        for (int e = 0; e < V; ++e) sa += r.v[e] * r.v[e];
        if constexpr (NB == 2) {
            const Row<V> q = branch_load<V>(B, row, c * V);
#pragma unroll
            for (int e = 0; e < V; ++e) sb += q.v[e] * q.v[e];
        }
    }
    float ra = A.g, rb = B.g;
    if (A.w) ra *= rsqrtf(cta_sum(sa, red[0]) / (float)W + eps);
    if (NB == 2 && B.w) rb *= rsqrtf(cta_sum(sb, red[1]) / (float)W + eps);
    float ss = 0.f;
    auto sum = [&](int c, const Row<V>& p, const Row<V>& q, Row<V>& r) {
#pragma unroll
        for (int e = 0; e < V; ++e) {
            r.v[e] += p.v[e] * ra * (A.w ? A.w[c * V + e] : 1.f);
            if constexpr (NB == 2) r.v[e] += q.v[e] * rb * (B.w ? B.w[c * V + e] : 1.f);
            ss += r.v[e] * r.v[e];
        }
        if constexpr (V == 4) store4(xr + c * 4, make_float4(r.v[0], r.v[1], r.v[2], r.v[3]));
        else xr[c] = r.v[0];
    };
#pragma unroll
    for (int k = 0; k < NK; ++k) {
        const int c = k * RS_THREADS + threadIdx.x;
        if (c < nc) sum(c, a[k], b[NB == 2 ? k : 0], xs[k]);
    }
    for (int c = kept + threadIdx.x; c < nc; c += RS_THREADS) {
        Row<V> p = branch_load<V>(A, row, c * V), q = p, r;
        if constexpr (NB == 2) q = branch_load<V>(B, row, c * V);
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = xr[c * V + e];
        sum(c, p, q, r);
    }
    if (!w) return;
    const float rs = rsqrtf(cta_sum(ss, red[2]) / (float)W + eps);
    T* o = out + row * W;
    auto put = [&](int c, const Row<V>& r) {
        if constexpr (V == 4) {
            const float4 m = *reinterpret_cast<const float4*>(w + c * 4);
            store4(o + c * 4, make_float4(r.v[0] * rs * m.x, r.v[1] * rs * m.y, r.v[2] * rs * m.z, r.v[3] * rs * m.w));
        } else from_f(o + c, r.v[0] * rs * w[c]);
    };
#pragma unroll
    for (int k = 0; k < NK; ++k) {
        const int c = k * RS_THREADS + threadIdx.x;
        if (c < nc) put(c, xs[k]);
    }
    for (int c = kept + threadIdx.x; c < nc; c += RS_THREADS) {
        Row<V> r;
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = xr[c * V + e];
        put(c, r);
    }
}

// The same for the many rows of a prompt (bf16 branches of one part each): persistent CTAs, the inputs of the rows ahead arrive by bulk
// copies in two stages of shared memory, the weights stay in registers.  W is a multiple of eight and at most 4 NK RS_THREADS.
template <int NB> __host__ __device__ constexpr int stream_row_bytes(int W) { return W * (4 + 2 * NB); }
template <int NK, int NB>
__global__ void __launch_bounds__(RS_THREADS) residual_norm_stream_kernel(const Branch A, const Branch B, float eps, float* __restrict__ x,
                                                                          const float* __restrict__ w, __nv_bfloat16* __restrict__ out, int n, int W,
                                                                          int* status) {
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ float red[4][32];
    __shared__ uint64_t bar[2];
    const int nc = W / 4, stage = (stream_row_bytes<NB>(W) + 127) & ~127;
    if (threadIdx.x == 0) {
        mbar_init(&bar[0], 1);
        mbar_init(&bar[1], 1);
        mbar_fence_init();
    }
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    auto load = [&](int row, int s) {
        unsigned char* d = smem + s * stage;
        mbar_expect_tx(&bar[s], (uint32_t)stream_row_bytes<NB>(W));
        bulk_g2s(d, x + (size_t)row * W, W * 4, &bar[s]);
        bulk_g2s(d + W * 4, (const __nv_bfloat16*)A.y + (size_t)row * A.ld, W * 2, &bar[s]);
        if constexpr (NB == 2) bulk_g2s(d + W * 6, (const __nv_bfloat16*)B.y + (size_t)row * B.ld, W * 2, &bar[s]);
    };
    if (threadIdx.x == 0) {
        load(blockIdx.x, 0);
        if ((int)(blockIdx.x + gridDim.x) < n) load(blockIdx.x + gridDim.x, 1);
    }
    const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
    float4 wa[NK], wb[NB == 2 ? NK : 1], wn[NK];
#pragma unroll
    for (int k = 0; k < NK; ++k) {
        const int c = k * RS_THREADS + threadIdx.x;
        wa[k] = c < nc && A.w ? load4<float>(A.w + c * 4) : one;
        if constexpr (NB == 2) wb[k] = c < nc && B.w ? load4<float>(B.w + c * 4) : one;
        wn[k] = c < nc ? load4<float>(w + c * 4) : one;
    }
    bool ok = true;
    int it = 0;
    for (int row = blockIdx.x; row < n; row += gridDim.x, ++it) {
        const int s = it & 1;
        if (ok) ok = mbar_wait(&bar[s], (uint32_t)((it >> 1) & 1), status);
        const float* xs_s = reinterpret_cast<const float*>(smem + s * stage);
        const __nv_bfloat16* a_s = reinterpret_cast<const __nv_bfloat16*>(smem + s * stage + W * 4);
        const __nv_bfloat16* b_s = reinterpret_cast<const __nv_bfloat16*>(smem + s * stage + W * 6);
        float4 a[NK], b[NB == 2 ? NK : 1];
        float ra = A.g, rb = B.g, sa = 0.f, sb = 0.f;
#pragma unroll
        for (int k = 0; k < NK; ++k) {
            const int c = k * RS_THREADS + threadIdx.x;
            if (c < nc) {
                a[k] = load4<__nv_bfloat16>(a_s + c * 4);
                sa += a[k].x * a[k].x + a[k].y * a[k].y + a[k].z * a[k].z + a[k].w * a[k].w;
                if constexpr (NB == 2) {
                    b[k] = load4<__nv_bfloat16>(b_s + c * 4);
                    sb += b[k].x * b[k].x + b[k].y * b[k].y + b[k].z * b[k].z + b[k].w * b[k].w;
                }
            }
        }
        if (A.w || (NB == 2 && B.w)) {
            sa = warp_sum(sa);
            if constexpr (NB == 2) sb = warp_sum(sb);
            if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sa; red[1][threadIdx.x >> 5] = sb; }
            __syncthreads();
            sa = sb = 0.f;
#pragma unroll
            for (int i = 0; i < RS_THREADS / 32; ++i) { sa += red[0][i]; sb += red[1][i]; }
            if (A.w) ra *= rsqrtf(sa / (float)W + eps);
            if (NB == 2 && B.w) rb *= rsqrtf(sb / (float)W + eps);
        }
        float ss = 0.f;
        float4 v[NK];
#pragma unroll
        for (int k = 0; k < NK; ++k) {
            const int c = k * RS_THREADS + threadIdx.x;
            if (c < nc) {
                float4 r = load4<float>(xs_s + c * 4);
                r.x += a[k].x * ra * wa[k].x; r.y += a[k].y * ra * wa[k].y; r.z += a[k].z * ra * wa[k].z; r.w += a[k].w * ra * wa[k].w;
                if constexpr (NB == 2) { r.x += b[k].x * rb * wb[k].x; r.y += b[k].y * rb * wb[k].y; r.z += b[k].z * rb * wb[k].z; r.w += b[k].w * rb * wb[k].w; }
                ss += r.x * r.x + r.y * r.y + r.z * r.z + r.w * r.w;
                store4(x + (size_t)row * W + c * 4, r);
                v[k] = r;
            }
        }
        ss = warp_sum(ss);
        if ((threadIdx.x & 31) == 0) red[2 + s][threadIdx.x >> 5] = ss;
        __syncthreads();                               // and the stage has been read
        if (threadIdx.x == 0 && ok && row + 2 * (int)gridDim.x < n) load(row + 2 * gridDim.x, s);
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < RS_THREADS / 32; ++i) ss += red[2 + s][i];
        const float rs = rsqrtf(ss / (float)W + eps);
#pragma unroll
        for (int k = 0; k < NK; ++k) {
            const int c = k * RS_THREADS + threadIdx.x;
            if (c < nc) store4(out + (size_t)row * W + c * 4, make_float4(v[k].x * rs * wn[k].x, v[k].y * rs * wn[k].y, v[k].z * rs * wn[k].z, v[k].w * rs * wn[k].w));
        }
    }
}

template <int NK, int NB>
static cudaError_t residual_norm_stream(const Branch& A, const Branch& B, float eps, float* x, const float* w, void* out, int n, int W, int* status,
                                        cudaStream_t st) {
    const int smem = 2 * ((stream_row_bytes<NB>(W) + 127) & ~127);
    auto k = residual_norm_stream_kernel<NK, NB>;
    cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, smem);
    if (e != cudaSuccess) return e;
    int dev = 0, sms = 0, per = 0;
    if ((e = cudaGetDevice(&dev)) != cudaSuccess) return e;
    if ((e = cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev)) != cudaSuccess) return e;
    if ((e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&per, k, RS_THREADS, smem)) != cudaSuccess) return e;
    return ptb_launch(k, dim3(std::min(n, sms * std::max(1, per))), dim3(RS_THREADS), (size_t)smem, st, ptb_pdl_enabled(), A, B, eps, x, w,
                      (__nv_bfloat16*)out, n, W, status);
}

template <typename T, int NB>
static cudaError_t residual_norm_launch(const Branch& A, const Branch& B, float eps, float* x, const float* w, void* out, int n, int W, bool vec,
                                        cudaStream_t st) {
    auto go = [&](auto k) { return ptb_launch(k, dim3(n), dim3(RS_THREADS), 0, st, ptb_pdl_enabled(), A, B, eps, x, w, (T*)out, W); };
    if (!vec) return go(residual_norm_kernel<T, 1, 4, NB>);
    const int nk = (W / 4 + RS_THREADS - 1) / RS_THREADS;
    if (nk <= 1) return go(residual_norm_kernel<T, 4, 1, NB>);
    if (nk <= 2) return go(residual_norm_kernel<T, 4, 2, NB>);
    return go(residual_norm_kernel<T, 4, 4, NB>);
}

}  // namespace ptb

using namespace ptb;

// x [n, W] fp32 += branch a (+ branch b, absent with yb null); h [n, W] (bf16 or fp32) = x / rms(x) * w unless w is null.  A branch: y in
// bf16 (f32 = 0) or as the sum of `splits` fp32 matrices `stride` apart, row pitch ld; times g; RMS-normed with the fp32 weight w[W]
// when that is given.  eps sits inside every root.  status: device int, set
// non-zero if a copy never arrived.
PTB_API int ptb_residual_norm(float* x, const void* ya, int f32a, int splits_a, long long stride_a, long long ld_a, const float* wa, float ga,
                              const void* yb, int f32b, int splits_b, long long stride_b, long long ld_b, const float* wb, float gb, float eps,
                              const float* w, void* h, int n, int W, int bf16, int* status, cudaStream_t st) {
    if (n <= 0) return 0;
    const Branch A{ya, f32a, splits_a, stride_a, ld_a, wa, ga}, B{yb, f32b, splits_b, stride_b, ld_b, wb, gb};
    const uintptr_t bases = (uintptr_t)x | (uintptr_t)ya | (uintptr_t)yb | (uintptr_t)wa | (uintptr_t)wb | (uintptr_t)w | (uintptr_t)h;
    const bool vec = W % 4 == 0 && (bases & 15) == 0 && ld_a % 4 == 0 && ld_b % 4 == 0 && stride_a % 4 == 0 && stride_b % 4 == 0;
    if (!ya || (splits_a > 1 && !f32a) || (splits_b > 1 && !f32b)) { ptb_set_error("residual_norm: partials are fp32, and the first branch is there"); return -1; }
    const bool stream = vec && bf16 && w && !f32a && !(yb && f32b) && n >= 1024 && W % 8 == 0 && ld_a % 8 == 0 && ld_b % 8 == 0 && W <= 16 * RS_THREADS;
    if (stream) {
        const bool small = W <= 8 * RS_THREADS;
        PTB_CUDA_OK((yb ? (small ? residual_norm_stream<2, 2> : residual_norm_stream<4, 2>) : (small ? residual_norm_stream<2, 1> : residual_norm_stream<4, 1>))(A, B, eps, x, w, h, n, W, status, st));
        return 0;
    }
    if (bf16) PTB_CUDA_OK((yb ? residual_norm_launch<__nv_bfloat16, 2> : residual_norm_launch<__nv_bfloat16, 1>)(A, B, eps, x, w, h, n, W, vec, st));
    else PTB_CUDA_OK((yb ? residual_norm_launch<float, 2> : residual_norm_launch<float, 1>)(A, B, eps, x, w, h, n, W, vec, st));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

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
