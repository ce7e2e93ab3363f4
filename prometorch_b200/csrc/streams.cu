// Several fp32 residual streams per token (hyper-connections) around layer-normed sublayers:
//   pair_embed_kernel   row = table[id] + pair table[(previous id * a + id * b) mod rows] + position table[pos], into every stream;
//   pair_tail_kernel    after a prompt pass: the last id of every sequence into its slot;
//   stream_step_kernel  what stands between two sublayers: the output of the one before (a product, split-K partials, the rows of its
//                       experts, a product beside them) times a sigmoid gate joins the streams through the connection's matrices, then
//                       the next sublayer's input is read off, normed and, one token per sequence, passed through the causal convolution
//                       of that sublayer's input.
// A slot, an id or a position outside its extent sets PTB_ERR_BOUNDS.
#include "common.cuh"
#include "ptb200_types.h"
#include <algorithm>

namespace ptb {
namespace streams {

constexpr int MAX_STREAMS = 16;
// Most threads of a row's CTA: a thread holds its columns of all streams in registers.
__host__ __device__ constexpr int max_threads(int S) { return S == 0 ? 256 : S > 2 ? 512 : 1024; }

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
template <typename T> __device__ __forceinline__ float rounded(float v) { return (float)(T)v; }

// ---------------------------------------------------------------------------------------------- into the streams
template <typename T, int V>
__global__ void __launch_bounds__(256) pair_embed_kernel(const __grid_constant__ PtbPairEmbed P) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = blockIdx.x;
    int id = P.ids[i * P.id_stride], pos = P.pos[i * P.pos_stride], slot = P.req[i * P.req_stride];
    bool bad = id < 0 || id >= P.V || pos < 0 || pos >= P.positions || slot < 0 || slot >= P.slots;
    long long before = -1;
    if (pos > 0 && slot >= 0 && slot < P.slots) {      // in a prompt pass the token before may be a row of the batch
        if (P.seqs && i > 0 && P.req[(i - 1) * P.req_stride] == slot) before = P.ids[(i - 1) * P.id_stride];
        else before = P.last[slot];
    }
    __syncthreads();                                   // every thread has read the slot
    if (!P.seqs && threadIdx.x == 0 && slot >= 0 && slot < P.slots) P.last[slot] = id;
    if (bad && threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
    id = min(max(id, 0), P.V - 1);
    pos = min(max(pos, 0), P.positions - 1);
    long long row = P.rows;                            // the row behind the hashed ones
    if (before >= 0) {
        row = (before * P.mul_before + (long long)id * P.mul_id) % P.rows;
        if (row < 0) row += P.rows;
    }
    const T *a = (const T*)P.table + (size_t)id * P.W, *b = (const T*)P.pairs + (size_t)row * P.W, *c = (const T*)P.at + (size_t)pos * P.W;
    float* x = P.x + i * P.streams * P.W;
    for (int e = threadIdx.x * V; e < P.W; e += blockDim.x * V) {
        Vals<V> v = ld<V>(a + e);
        const Vals<V> p = ld<V>(b + e), q = ld<V>(c + e);
#pragma unroll
        for (int k = 0; k < V; ++k) v.v[k] += p.v[k] + q.v[k];
        for (int s = 0; s < P.streams; ++s) st<V>(x + (size_t)s * P.W + e, v);
    }
}

__global__ void __launch_bounds__(256) pair_tail_kernel(const __grid_constant__ PtbPairEmbed P) {
    pdl_wait();
    pdl_launch_dependents();
    const int i = blockIdx.x * blockDim.x + threadIdx.x;
    if (i >= P.n_seqs) return;
    const int4 s = reinterpret_cast<const int4*>(P.seqs)[i];       // first row, rows, position of the first, slot
    if (s.w < 0 || s.w >= P.slots || s.x < 0 || s.y < 1 || s.x + s.y > P.n) return;
    P.last[s.w] = P.ids[(size_t)(s.x + s.y - 1) * P.id_stride];
}

// ---------------------------------------------------------------------------------------------- between two sublayers
__device__ __forceinline__ float cta_total(float v, float* red) {
    v = warp_sum(v);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = v;
    __syncthreads();
    const float t = (threadIdx.x & 31) < (blockDim.x >> 5) ? red[threadIdx.x & 31] : 0.f;
    return warp_sum(t);
}

template <typename T, int V>
__device__ __forceinline__ Vals<V> dense_load(const PtbDense& D, size_t row, int c) {
    Vals<V> r;
    if (D.f32) {
        const float* p = (const float*)D.y + row * D.ld + c;
        r = ld<V>(p);
#pragma unroll 4
        for (int s = 1; s < D.splits; ++s) {
            const Vals<V> t = ld<V>(p + s * D.stride);
#pragma unroll
            for (int e = 0; e < V; ++e) r.v[e] += t.v[e];
        }
    } else r = ld<V>((const __nv_bfloat16*)D.y + row * D.ld + c);
    return r;
}

// One CTA per row.  T: the compute type; V elements per access; S streams (0: any number up to MAX_STREAMS).
template <typename T, int V, int S>
__global__ void __launch_bounds__(max_threads(S)) stream_step_kernel(const __grid_constant__ PtbStreamStep P) {
    extern __shared__ __align__(16) float u_s[];       // [W] what the next sublayer reads
    __shared__ float mix_s[MAX_STREAMS * MAX_STREAMS], out_s[MAX_STREAMS], in_s[MAX_STREAMS], red[2][32];
    const int streams = S ? S : P.streams, W = P.W;
    for (int e = threadIdx.x; e < streams * streams; e += blockDim.x) {      // weights of the model: no kernel before this one writes them
        if (P.mix) mix_s[e] = P.mix[e];
        if (e < streams) {
            if (P.way_out) out_s[e] = P.way_out[e];
            in_s[e] = P.way_in ? P.way_in[e] : 1.f;
        }
    }
    pdl_wait();
    pdl_launch_dependents();
    __syncthreads();
    const size_t o = blockIdx.x;
    long long row = P.index ? P.index[o] : (long long)o;
    if (row < 0 || row >= P.n) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        row = 0;
    }
    float* x = P.x + (size_t)row * streams * W;
    float sum = 0.f;
    constexpr int SC = S ? S : MAX_STREAMS;
#pragma unroll 2
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        Vals<V> xs[SC], u;
#pragma unroll
        for (int s = 0; s < SC; ++s)
            if (s < streams) xs[s] = ld<V>(x + (size_t)s * W + c);
#pragma unroll
        for (int e = 0; e < V; ++e) u.v[e] = 0.f;
        if (P.mix) {
            Vals<V> y;
            const Vals<V> g = dense_load<T, V>(P.gate, row, c), b = ld<V>(P.gate_bias + c);
            if (P.y.y) y = dense_load<T, V>(P.y, row, c);
            else {
#pragma unroll
                for (int e = 0; e < V; ++e) y.v[e] = 0.f;
            }
            if (P.index_of) {
#pragma unroll 4
                for (int k = 0; k < P.top; ++k) {
                    int r = P.index_of[(size_t)row * P.top + k];
                    const float f = P.weight[(size_t)row * P.top + k];
                    if (r >= P.e_rows || r < -1) {
                        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
                        r = -1;
                    }
                    const T* src = r < 0 ? (const T*)P.self + (size_t)row * W : (const T*)P.experts + (size_t)r * P.e_ld;
                    const Vals<V> t = ld<V>(src + c);
#pragma unroll
                    for (int e = 0; e < V; ++e) y.v[e] = fmaf(f, t.v[e], y.v[e]);
                }
            }
#pragma unroll
            for (int e = 0; e < V; ++e) y.v[e] *= sigmoid(g.v[e] + b.v[e]);
#pragma unroll
            for (int t = 0; t < SC; ++t)
                if (t < streams) {
                    Vals<V> z;
#pragma unroll
                    for (int e = 0; e < V; ++e) z.v[e] = out_s[t] * y.v[e];
#pragma unroll
                    for (int s = 0; s < SC; ++s)
                        if (s < streams) {
                            const float m = mix_s[s * streams + t];
#pragma unroll
                            for (int e = 0; e < V; ++e) z.v[e] = fmaf(m, xs[s].v[e], z.v[e]);
                        }
                    st<V>(x + (size_t)t * W + c, z);
#pragma unroll
                    for (int e = 0; e < V; ++e) u.v[e] = fmaf(in_s[t], z.v[e], u.v[e]);
                }
        } else {
#pragma unroll
            for (int t = 0; t < SC; ++t)
                if (t < streams)
#pragma unroll
                    for (int e = 0; e < V; ++e) u.v[e] = fmaf(in_s[t], xs[t].v[e], u.v[e]);
        }
        if (P.norm) {
            st<V>(u_s + c, u);
#pragma unroll
            for (int e = 0; e < V; ++e) sum += u.v[e];
        }
    }
    if (!P.norm) return;
    const float mean = cta_total(sum, red[0]) / (float)W;
    float var = 0.f;
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        const Vals<V> u = ld<V>(u_s + c);
#pragma unroll
        for (int e = 0; e < V; ++e) { const float d = u.v[e] - mean; var = fmaf(d, d, var); }
    }
    const float rs = rsqrtf(cta_total(var, red[1]) / (float)W + P.eps);
    T *h = (T*)P.h + o * W, *hc = P.conv ? (T*)P.conv_out + o * W : nullptr;
    int pos = 0, slot = -1;
    if (P.conv) {
        pos = P.pos[(size_t)o * P.pos_stride];
        slot = P.req[(size_t)o * P.req_stride];
        if (slot < 0 || slot >= P.slots) {
            if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
            slot = -1;
        }
    }
    for (int c = threadIdx.x * V; c < W; c += blockDim.x * V) {
        Vals<V> u = ld<V>(u_s + c);
        const Vals<V> w = ld<V>(P.norm + c);
#pragma unroll
        for (int e = 0; e < V; ++e) u.v[e] = rounded<T>((u.v[e] - mean) * rs * w.v[e]);
        st<V>(h + c, u);
        if (!hc) continue;
        // this thread alone touches these channels of the slot: it reads the inputs before this token and shifts them
        Vals<V> a = ld<V>(P.conv + (size_t)(P.taps - 1) * W + c);
#pragma unroll
        for (int e = 0; e < V; ++e) a.v[e] = fmaf(a.v[e], u.v[e], u.v[e]);
        T* state = (T*)P.conv_state + (size_t)max(slot, 0) * (P.taps - 1) * W + c;
        for (int m = P.taps - 1; m >= 1; --m) {
            if (pos - m < 0 || slot < 0) continue;     // before the sequence's start
            const Vals<V> t = ld<V>(state + (size_t)(P.taps - 1 - m) * W), k = ld<V>(P.conv + (size_t)(P.taps - 1 - m) * W + c);
#pragma unroll
            for (int e = 0; e < V; ++e) a.v[e] = fmaf(k.v[e], t.v[e], a.v[e]);
            if (m < P.taps - 1) st<V>(state + (size_t)(P.taps - 2 - m) * W, t);
        }
        if (slot >= 0 && P.taps > 1) st<V>(state + (size_t)(P.taps - 2) * W, u);
        st<V>(hc + c, a);
    }
}

template <typename T, int V>
static cudaError_t step_launch(const PtbStreamStep& p, cudaStream_t s) {
    const int lanes = (p.W + V - 1) / V, most = p.m <= 256 ? max_threads(p.streams > 4 ? 0 : p.streams) : 256;
    const int threads = std::min(most, (lanes + 31) / 32 * 32);
    const size_t smem = p.norm ? (size_t)p.W * 4 : 0;
    auto go = [&](auto k) {
        if (smem > 40 * 1024) {
            const cudaError_t e = cudaFuncSetAttribute(k, cudaFuncAttributeMaxDynamicSharedMemorySize, 220 * 1024);
            if (e != cudaSuccess) return e;
        }
        return ptb_launch(k, dim3(p.m), dim3(threads), smem, s, ptb_pdl_enabled(), p);
    };
    switch (p.streams) {
        case 1: return go(stream_step_kernel<T, V, 1>);
        case 2: return go(stream_step_kernel<T, V, 2>);
        case 3: return go(stream_step_kernel<T, V, 3>);
        case 4: return go(stream_step_kernel<T, V, 4>);
        default: return go(stream_step_kernel<T, 1, 0>);
    }
}

}  // namespace streams
}  // namespace ptb

using namespace ptb;

// x [n][streams][W] fp32: every stream of token i is table[id] + pairs[row] + at[pos]; see PtbPairEmbed.
PTB_API int ptb_pair_embed(const PtbPairEmbed* args, cudaStream_t s) {
    const PtbPairEmbed& p = *args;
    if (p.n <= 0) return 0;
    if (!p.table || !p.pairs || !p.at || !p.last || p.rows < 1 || p.V < 1 || p.positions < 1 || p.W < 1 || p.streams < 1) {
        ptb_set_error("pair_embed: missing table, or %d rows, %d ids, %d positions", p.rows, p.V, p.positions);
        return -1;
    }
    const bool pdl = ptb_pdl_enabled();
    const bool vec = p.W % 4 == 0 && (((uintptr_t)p.table | (uintptr_t)p.pairs | (uintptr_t)p.at | (uintptr_t)p.x) & 15) == 0;
    auto kern = p.bf16 ? (vec ? streams::pair_embed_kernel<__nv_bfloat16, 4> : streams::pair_embed_kernel<__nv_bfloat16, 1>)
                       : (vec ? streams::pair_embed_kernel<float, 4> : streams::pair_embed_kernel<float, 1>);
    PTB_CUDA_OK(ptb_launch(kern, dim3(p.n), dim3(256), 0, s, pdl, p));
    if (p.seqs && p.n_seqs > 0) PTB_CUDA_OK(ptb_launch(streams::pair_tail_kernel, dim3((p.n_seqs + 255) / 256), dim3(256), 0, s, pdl, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// The step between two sublayers of a decoder with several residual streams; see PtbStreamStep.
PTB_API int ptb_stream_step(const PtbStreamStep* args, cudaStream_t s) {
    const PtbStreamStep& p = *args;
    if (p.m <= 0) return 0;
    if (p.streams < 1 || p.streams > streams::MAX_STREAMS || p.W < 1 || p.W > 55 * 1024) {
        ptb_set_error("stream_step: %d streams (at most %d) of %d columns", p.streams, streams::MAX_STREAMS, p.W);
        return -1;
    }
    if ((p.mix && (!p.gate.y || !p.gate_bias || !p.way_out || p.index || p.m != p.n || (p.index_of && (!p.weight || !p.self || !p.experts)))) ||
        (p.norm && !p.h) || (p.conv && (!p.conv_out || !p.pos || !p.req || p.taps < 1 || (p.taps > 1 && !p.conv_state))) || (p.y.splits > 1 && !p.y.f32) ||
        (p.gate.splits > 1 && !p.gate.f32)) {
        ptb_set_error("stream_step: missing operand");
        return -1;
    }
    const uintptr_t bases = (uintptr_t)p.x | (uintptr_t)p.y.y | (uintptr_t)p.gate.y | (uintptr_t)p.gate_bias | (uintptr_t)p.norm | (uintptr_t)p.h | (uintptr_t)p.conv |
                            (uintptr_t)p.conv_out | (uintptr_t)p.conv_state | (uintptr_t)p.self | (uintptr_t)p.experts;
    const bool vec = p.W % 4 == 0 && p.y.ld % 4 == 0 && p.y.stride % 4 == 0 && p.gate.ld % 4 == 0 && p.gate.stride % 4 == 0 && p.e_ld % 4 == 0 && (bases & 15) == 0;
    if (p.bf16) PTB_CUDA_OK((vec ? streams::step_launch<__nv_bfloat16, 4>(p, s) : streams::step_launch<__nv_bfloat16, 1>(p, s)));
    else PTB_CUDA_OK((vec ? streams::step_launch<float, 4>(p, s) : streams::step_launch<float, 1>(p, s)));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
