// Attention whose weights are an element-wise function of the score instead of a softmax over the keys ("gated" attention), over
// the paged cache.  What a design can set: the score's scale, a soft cap, an additive bias per head and distance (table lookup,
// the last entry stands for everything farther), a sliding window, and a mixing matrix that makes every head's weight a linear
// combination of all heads' weights of the same query and key:
//     s_h(i, j)  = cap * tanh(scale * q_h(i) . k_g(h)(j) / cap) + bias[h][min(i - j, nb - 1)]
//     w_h(i, j)  = sigmoid(s_h(i, j))           for 0 <= i - j < window
//     o_h(i)     = sum_j (sum_f talk[h][f] w_f(i, j)) v_g(h)(j)
// The weights are not normalised, so partial results over disjoint keys simply add.
#pragma once
#include "common.cuh"

namespace ptb {

constexpr int GA_PAGE = 64;            // tokens per cache page
constexpr int GA_KEYS = 128;           // most keys one CTA of the row kernels handles

struct GatedAttnParams {
    const void* q;                     // [n, H, Dp]
    void* out;                         // [n, H * Dv]
    float* work;                       // [n, nsplit, H, Dvp] partial sums when nsplit > 1
    const int* pos;                    // position of row i at pos[i * pos_stride]
    const int* req;                    // its row of the page table at req[i * req_stride]
    const int* page_table;
    const void* k_pages;               // [n_pages, G, 64, Dp]
    const void* v_pages;               // [n_pages, G, 64, Dvp]
    const float* bias;                 // [H, nb]
    const float* talk;                 // [H, H] (to head, from head), or null
    int pos_stride, req_stride, pt_stride, n_pages;
    int n, H, G, Dp, Dv, Dvp, nb, window, nsplit, kcap;
    float scale, cap, inv_cap;         // cap 0: no cap
    int* status;
};

// tanh without the cancellation of 1 - 2 / (exp + 1) near zero: there, its Taylor series through x^15 (below 0.5 the next term is
// smaller than 1e-8 of the value).
constexpr float TANH_SERIES_MAX = 0.5f;
__device__ __forceinline__ float tanh_series(float x) {
    const float u = x * x;
    float p = -929569.f / 638512875.f;
    p = fmaf(p, u, 21844.f / 6081075.f);
    p = fmaf(p, u, -1382.f / 155925.f);
    p = fmaf(p, u, 62.f / 2835.f);
    p = fmaf(p, u, -17.f / 315.f);
    p = fmaf(p, u, 2.f / 15.f);
    p = fmaf(p, u, -1.f / 3.f);
    return fmaf(x * u, p, x);
}
__device__ __forceinline__ float tanh_any(float x) {
    const float ax = fabsf(x), e = copysignf(1.f - __fdividef(2.f, __expf(2.f * fminf(ax, 40.f)) + 1.f), x);
    return ax < TANH_SERIES_MAX ? tanh_series(x) : e;
}
__device__ __forceinline__ float soft_cap(float s, float cap, float inv_cap) { return cap * tanh_any(s * inv_cap); }
// 1 / (1 + 2^z): with z = -s log2(e) the sigmoid of s; 2^z may overflow to infinity, whose reciprocal is 0.
__device__ __forceinline__ float sigmoid_ex2(float z) {
    float e, r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(e) : "f"(z));
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + e));
    return r;
}
__device__ __forceinline__ float sigmoid_w(float s) { return __fdividef(1.f, 1.f + __expf(fminf(-s, 80.f))); }

__device__ __forceinline__ float gated_weight(const GatedAttnParams& P, float dot, int h, int dist) {
    float s = dot * P.scale;
    if (P.cap > 0.f) s = soft_cap(s, P.cap, P.inv_cap);
    return sigmoid_w(s + __ldg(P.bias + (size_t)h * P.nb + min(dist, P.nb - 1)));
}

}  // namespace ptb
