// Recurrent layers with a matrix state S [D, Dv] per head and sequence, fp32:
//   decay attention   S <- decay_h S + k v^T;  o = S^T q
//   gated delta rule  S <- g S (g per key channel, or one number);  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q
// with g = exp(-rate_h softplus(a + dt_bias)), beta a sigmoid, q and k unit vectors (q also times D^-1/2);
//   state-space step  S <- exp(-rate_h dt) S + dt k v^T;  o = S^T q + skip_h v,  dt = softplus(a + dt_bias) per head, q and k per group of heads.
#pragma once
#include "common.cuh"
#include "ptb200_types.h"

namespace ptb {

template <typename T> __device__ __forceinline__ float rc_f(T v);
template <> __device__ __forceinline__ float rc_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float rc_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T rc_t(float v);
template <> __device__ __forceinline__ float rc_t<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 rc_t<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// max(x, 0) + log(1 + z) with z = exp(-|x|) <= 1, by log(1 + z) = 2 artanh(s), s = z / (2 + z) <= 1/3, and the series of artanh through
// s^13 (the next term is below 1e-8 of the sum).
__device__ __forceinline__ float softplus(float x) {
    const float z = __expf(-fabsf(x)), s = __fdividef(z, 2.f + z), q = s * s;
    float p = fmaf(q, 1.f / 13.f, 1.f / 11.f);
    p = fmaf(q, p, 1.f / 9.f); p = fmaf(q, p, 1.f / 7.f); p = fmaf(q, p, 1.f / 5.f); p = fmaf(q, p, 1.f / 3.f);
    return fmaxf(x, 0.f) + 2.f * s * fmaf(q, p, 1.f);
}
// log of the decay of one head's key channel
__device__ __forceinline__ float delta_log_decay(float a, float dt, float rate) { return -rate * softplus(a + dt); }

constexpr float UNIT_EPS = 1e-6f;

// The rows of one sequence in the batch: `count` rows from row0, the first at position pos0, state slot `slot` (-1: out of range).
struct Span { int row0, count, pos0, slot; };
__device__ __forceinline__ Span span_of(const PtbRecurrence& P, int i) {
    Span s;
    if (P.seqs) {
        const int4 v = reinterpret_cast<const int4*>(P.seqs)[i];
        s = Span{v.x, v.y, v.z, v.w};
        if (s.row0 < 0 || s.count < 0 || s.row0 + s.count > P.n) s = Span{0, 0, 0, -1};
    } else {
        s = Span{i, 1, P.pos[(size_t)i * P.pos_stride], P.req[(size_t)i * P.req_stride]};
    }
    if (s.slot < 0 || s.slot >= P.slots) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        s.slot = -1;
    }
    return s;
}

}  // namespace ptb
