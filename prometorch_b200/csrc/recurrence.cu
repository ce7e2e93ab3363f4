// Recurrent layers token by token, and what surrounds them:
//   short_conv_kernel / conv_tail_kernel   causal convolution over time per channel, then SiLU, or the input added; the last inputs stay in the
//                                          sequence's slot;
//   recurrence_kernel                      one CTA per (32 value columns, head, sequence); the state stays in registers from the first
//                                          token to the last.  One token per sequence in a decode pass, every token of a prompt in
//                                          true fp32 arithmetic (recurrence_chunk.cu has the matrix form for bf16 prompts);
//   group_norm_gate_kernel                 RMS norm of groups of columns, weight, sigmoid or SiLU gate (behind the norm, or ahead of it).
// A slot outside its extent sets PTB_ERR_BOUNDS and its sequence is skipped.
#include "recurrence.cuh"
#include <algorithm>

namespace ptb {

// ---------------------------------------------------------------------------------------------- short convolution
struct ConvParams {
    const void* x;
    long long ld;
    const float* w;                    // [taps][C]
    const float* bias;                 // [C] or null
    int add;                           // the result is the input plus the convolution, without SiLU
    void* state;                       // [slots][taps - 1][C]
    void* out;                         // [n][C]
    const int* pos;
    const int* req;
    const int4* seqs;                  // null: one token per row
    int C, taps, n, slots, pos_stride, req_stride, n_seqs;
    int* status;
};
template <typename T, int E> struct Elems { float v[E]; };
template <typename T, int E>
__device__ __forceinline__ Elems<T, E> ld_elems(const T* p) {
    Elems<T, E> r;
    if constexpr (E == 8 && sizeof(T) == 2) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); r.v[2 * i] = f.x; r.v[2 * i + 1] = f.y; }
    } else if constexpr (E == 4 && sizeof(T) == 2) {
        const uint2 raw = *reinterpret_cast<const uint2*>(p);
        const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.x)), b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&raw.y));
        r.v[0] = a.x; r.v[1] = a.y; r.v[2] = b.x; r.v[3] = b.y;
    } else if constexpr (E % 4 == 0 && sizeof(T) == 4) {
#pragma unroll
        for (int i = 0; i < E; i += 4) {
            const float4 f = *reinterpret_cast<const float4*>(p + i);
            r.v[i] = f.x; r.v[i + 1] = f.y; r.v[i + 2] = f.z; r.v[i + 3] = f.w;
        }
    } else {
#pragma unroll
        for (int i = 0; i < E; ++i) r.v[i] = rc_f<T>(p[i]);
    }
    return r;
}
template <typename T, int E>
__device__ __forceinline__ void st_elems(T* p, const Elems<T, E>& r) {
    if constexpr (E == 8 && sizeof(T) == 2) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(r.v[2 * i], r.v[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    } else if constexpr (E == 4 && sizeof(T) == 2) {
        const __nv_bfloat162 a = __floats2bfloat162_rn(r.v[0], r.v[1]), b = __floats2bfloat162_rn(r.v[2], r.v[3]);
        *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
    } else if constexpr (E % 4 == 0 && sizeof(T) == 4) {
#pragma unroll
        for (int i = 0; i < E; i += 4) *reinterpret_cast<float4*>(p + i) = make_float4(r.v[i], r.v[i + 1], r.v[i + 2], r.v[i + 3]);
    } else {
#pragma unroll
        for (int i = 0; i < E; ++i) p[i] = rc_t<T>(r.v[i]);
    }
}

constexpr int CONV_TOKENS = 16;        // consecutive rows of one thread of a prompt pass

// Inputs of the channels c.. that lie `m` tokens before row i (m <= taps - 1), of which `in_batch` are rows of the batch.
template <typename T, int E>
__device__ __forceinline__ Elems<T, E> conv_input(const ConvParams& P, int i, int m, int in_batch, int pos, int slot, int c) {
    if (m <= in_batch) return ld_elems<T, E>((const T*)P.x + (size_t)(i - m) * P.ld + c);
    Elems<T, E> z;
#pragma unroll
    for (int e = 0; e < E; ++e) z.v[e] = 0.f;
    if (pos - m < 0 || slot < 0) return z;
    return ld_elems<T, E>((const T*)P.state + ((size_t)slot * (P.taps - 1) + (P.taps - 1 - (m - in_batch))) * P.C + c);
}

template <int E>
__device__ __forceinline__ void conv_bias(const ConvParams& P, int c, Elems<float, E>& b) {
    if (P.bias) b = ld_elems<float, E>(P.bias + c);
    else {
#pragma unroll
        for (int e = 0; e < E; ++e) b.v[e] = 0.f;
    }
}

// A prompt pass with a fixed number of taps: weights and the last inputs stay in registers while a thread walks its rows.
template <typename T, int E, int TAPS>
__global__ void __launch_bounds__(256) short_conv_taps_kernel(const __grid_constant__ ConvParams P) {
    pdl_wait();
    pdl_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * E;
    if (c >= P.C) return;
    const int lo = blockIdx.y * CONV_TOKENS, hi = min(lo + CONV_TOKENS, P.n);
    Elems<float, E> w[TAPS], x[TAPS], bias;            // x[m]: the input m tokens back
    conv_bias(P, c, bias);
#pragma unroll
    for (int m = 0; m < TAPS; ++m) w[m] = ld_elems<float, E>(P.w + (size_t)(TAPS - 1 - m) * P.C + c);
    int before = -1;                                   // slot of the row before
#pragma unroll 4
    for (int i = lo; i < hi; ++i) {
        int slot = P.req[(size_t)i * P.req_stride];
        const Elems<T, E> now = ld_elems<T, E>((const T*)P.x + (size_t)i * P.ld + c);
        if (slot < 0 || slot >= P.slots) {
            if (P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
            slot = -1;
        }
        if (i == lo || slot != before) {               // a sequence starts here, or this thread's rows do
            const int pos = P.pos[(size_t)i * P.pos_stride];
            int in_batch = 0;
            while (in_batch < TAPS - 1 && i - in_batch - 1 >= 0 && P.req[(size_t)(i - in_batch - 1) * P.req_stride] == slot) ++in_batch;
#pragma unroll
            for (int m = 1; m < TAPS; ++m) {
                const Elems<T, E> v = conv_input<T, E>(P, i, m, in_batch, pos, slot, c);
#pragma unroll
                for (int e = 0; e < E; ++e) x[m].v[e] = v.v[e];
            }
            before = slot;
        }
        Elems<T, E> acc;
#pragma unroll
        for (int e = 0; e < E; ++e) {
            x[0].v[e] = now.v[e];
            float a = x[TAPS - 1].v[e] * w[TAPS - 1].v[e];
#pragma unroll
            for (int m = TAPS - 2; m >= 0; --m) a = fmaf(x[m].v[e], w[m].v[e], a);
            a += bias.v[e];
            acc.v[e] = P.add ? now.v[e] + a : silu(a);
#pragma unroll
            for (int m = TAPS - 1; m > 0; --m) x[m].v[e] = x[m - 1].v[e];
        }
        st_elems<T, E>((T*)P.out + (size_t)i * P.C + c, acc);
    }
}

template <typename T, int E>
__global__ void __launch_bounds__(256) short_conv_kernel(const __grid_constant__ ConvParams P) {
    pdl_wait();
    pdl_launch_dependents();
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * E;
    if (c >= P.C) return;
    const int per = P.seqs ? CONV_TOKENS : 1, lo = blockIdx.y * per, hi = min(lo + per, P.n);
    Elems<float, E> bias;
    conv_bias(P, c, bias);
    for (int i = lo; i < hi; ++i) {
        const int pos = P.pos[(size_t)i * P.pos_stride];
        int slot = P.req[(size_t)i * P.req_stride], in_batch = 0;
        if (P.seqs)
            while (in_batch < P.taps - 1 && i - in_batch - 1 >= 0 && P.req[(size_t)(i - in_batch - 1) * P.req_stride] == slot) ++in_batch;
        if (slot < 0 || slot >= P.slots) {
            if (P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
            slot = -1;
        }
        const Elems<T, E> now = ld_elems<T, E>((const T*)P.x + (size_t)i * P.ld + c);
        Elems<T, E> acc;
        {
            const Elems<float, E> w = ld_elems<float, E>(P.w + (size_t)(P.taps - 1) * P.C + c);
#pragma unroll
            for (int e = 0; e < E; ++e) acc.v[e] = fmaf(now.v[e], w.v[e], bias.v[e]);
        }
        T* st = (T*)P.state + (size_t)max(slot, 0) * (P.taps - 1) * P.C + c;
        for (int m = P.taps - 1; m >= 1; --m) {
            const Elems<T, E> x = conv_input<T, E>(P, i, m, in_batch, pos, slot, c);
            const Elems<float, E> w = ld_elems<float, E>(P.w + (size_t)(P.taps - 1 - m) * P.C + c);
#pragma unroll
            for (int e = 0; e < E; ++e) acc.v[e] = fmaf(x.v[e], w.v[e], acc.v[e]);
            // one token per row: this thread alone touches these channels of the slot, so it shifts them here
            if (!P.seqs && slot >= 0 && m < P.taps - 1) st_elems<T, E>(st + (size_t)(P.taps - 2 - m) * P.C, x);
        }
        if (!P.seqs && slot >= 0 && P.taps > 1) st_elems<T, E>(st + (size_t)(P.taps - 2) * P.C, now);
#pragma unroll
        for (int e = 0; e < E; ++e) acc.v[e] = P.add ? now.v[e] + acc.v[e] : silu(acc.v[e]);
        st_elems<T, E>((T*)P.out + (size_t)i * P.C + c, acc);
    }
}

// After a prompt pass: the last taps - 1 inputs of every sequence into its slot.
template <typename T>
__global__ void __launch_bounds__(256) conv_tail_kernel(const __grid_constant__ ConvParams P) {
    pdl_wait();
    pdl_launch_dependents();
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int4 s = P.seqs[blockIdx.y];                 // row0, count, pos0, slot
    if (c >= P.C || s.w < 0 || s.w >= P.slots || s.x < 0 || s.y < 0 || s.x + s.y > P.n) return;
    T* st = (T*)P.state + (size_t)s.w * (P.taps - 1) * P.C + c;
    for (int j = 0; j < P.taps - 1; ++j) {
        const int r = s.y - (P.taps - 1) + j;          // row of the sequence in the batch; before it: the old slot, shifted
        T v = rc_t<T>(0.f);
        if (r >= 0) v = ((const T*)P.x)[(size_t)(s.x + r) * P.ld + c];
        else if (s.z + r >= 0) v = st[(size_t)(j + s.y) * P.C];
        st[(size_t)j * P.C] = v;
    }
}

// ---------------------------------------------------------------------------------------------- token by token
constexpr int RC_THREADS = 256, RC_WARPS = 8, RC_COLS = 32;

// Thread (tx, ty): value columns v0 + 4 tx .. + 3, state rows ty, ty + 32, ...  One barrier per token: the next token's vectors are
// staged, and this token's partial sums left, in buffers that alternate.
// MODE: `delta` of PtbRecurrence.
template <typename T, int MODE, int RM>
__global__ void __launch_bounds__(RC_THREADS) recurrence_kernel(const __grid_constant__ PtbRecurrence P) {
    constexpr bool DELTA = MODE == 1 || MODE == 2;
    __shared__ float q_s[3][RM * 32], k_s[3][RM * 32], g_s[3][MODE == 1 ? RM * 32 : 2];      // three: a slow warp may still update with the token before
    __shared__ float red_s[2][RC_WARPS][4];
    __shared__ float4 part_s[2][RC_WARPS][8][2];
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, v0 = blockIdx.x * RC_COLS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, tx = lane & 7, ty = threadIdx.x >> 3;
    const Span s = span_of(P, blockIdx.z);
    if (s.slot < 0 || s.count == 0) return;
    const int D = P.D, Dv = P.Dv, hk = h / (P.H / P.G), col = v0 + tx * 4;
    const int live = max(0, min(4, Dv - col));
    const bool vec = (Dv & 3) == 0;
    float* st = P.state + (((size_t)s.slot * P.H + h) * D) * Dv;
    float S[RM][4];
#pragma unroll
    for (int i = 0; i < RM; ++i) {
        const int d = ty + 32 * i;
#pragma unroll
        for (int e = 0; e < 4; ++e) S[i][e] = 0.f;
        if (s.pos0 > 0 && d < D && live > 0) {
            if (vec) {
                const float4 t = *reinterpret_cast<const float4*>(st + (size_t)d * Dv + col);
                S[i][0] = t.x; S[i][1] = t.y; S[i][2] = t.z; S[i][3] = t.w;
            } else
                for (int e = 0; e < live; ++e) S[i][e] = st[(size_t)d * Dv + col + e];
        }
    }
    const float rate = P.decay[h], skip = MODE == 3 ? P.skip[h] : 0.f;
    auto stage = [&](int i) {
        const int b = i % 3;
        const T* row = (const T*)P.x + (size_t)(s.row0 + i) * P.ld;
        float qq = 0.f, kk = 0.f, qk = 0.f;
        for (int d = threadIdx.x; d < RM * 32; d += RC_THREADS) {
            float q = 0.f, k = 0.f, g = rate;
            if (d < D) {
                q = rc_f<T>(row[P.q_col + hk * D + d]);
                k = rc_f<T>(row[P.k_col + hk * D + d]);
                if constexpr (MODE == 1) g = expf(delta_log_decay(((const float*)P.a)[(size_t)(s.row0 + i) * P.ld_a + h * D + d], P.dt_bias[h * D + d], rate));
                else if (MODE == 0 && P.silu) { q = silu(q); k = silu(k); }
            }
            q_s[b][d] = q; k_s[b][d] = k;
            if constexpr (MODE == 1) g_s[b][d] = g;
            qq += q * q; kk += k * k; qk += q * k;
        }
        qq = warp_sum(qq); kk = warp_sum(kk); qk = warp_sum(qk);
        if constexpr (MODE == 3)
            if (threadIdx.x == 0) {                    // the decay and the step
                const float dt = softplus(rc_f<T>(((const T*)P.a)[(size_t)(s.row0 + i) * P.ld_a + h]) + P.dt_bias[h]);
                g_s[b][0] = expf(-rate * dt);
                g_s[b][1] = dt;
            }
        if constexpr (MODE == 2)
            if (threadIdx.x == 0) g_s[b][0] = expf(delta_log_decay(rc_f<T>(((const T*)P.a)[(size_t)(s.row0 + i) * P.ld_a + h]), P.dt_bias[h], rate));
        if (lane == 0) { red_s[i & 1][warp][0] = qq; red_s[i & 1][warp][1] = kk; red_s[i & 1][warp][2] = qk; }
    };
    stage(0);
    __syncthreads();
    for (int i = 0; i < s.count; ++i) {
        const int b = i & 1, c = i % 3;
        const size_t r = (size_t)(s.row0 + i);
        float v[4] = {0.f, 0.f, 0.f, 0.f}, beta = 1.f;
        for (int e = 0; e < live; ++e) {
            v[e] = rc_f<T>(((const T*)P.x)[r * P.ld + P.v_col + (size_t)h * Dv + col + e]);
            if (MODE == 0 && P.silu) v[e] = silu(v[e]);
        }
        if constexpr (DELTA) beta = sigmoid(rc_f<T>(((const T*)P.beta)[r * P.ld_beta + h]));
        float qq = 0.f, kk = 0.f, qk = 0.f;
#pragma unroll
        for (int w = 0; w < RC_WARPS; ++w) { qq += red_s[b][w][0]; kk += red_s[b][w][1]; qk += red_s[b][w][2]; }
        const float qn = DELTA ? rsqrtf(qq + UNIT_EPS) * rsqrtf((float)D) : 1.f, kn = DELTA ? rsqrtf(kk + UNIT_EPS) : 1.f;
        float sk[4] = {0.f, 0.f, 0.f, 0.f}, sq[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
        for (int j = 0; j < RM; ++j) {
            const int d = ty + 32 * j;
            const float g = MODE == 1 ? g_s[c][d] : MODE >= 2 ? g_s[c][0] : rate, k = k_s[c][d], q = q_s[c][d];
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                S[j][e] *= g;
                if constexpr (DELTA) sk[e] = fmaf(S[j][e], k, sk[e]);
                sq[e] = fmaf(S[j][e], q, sq[e]);
            }
        }
#pragma unroll
        for (int o = 8; o <= 16; o <<= 1)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                if constexpr (DELTA) sk[e] += __shfl_xor_sync(0xffffffffu, sk[e], o);
                sq[e] += __shfl_xor_sync(0xffffffffu, sq[e], o);
            }
        if (lane < 8) {
            if constexpr (DELTA) part_s[b][warp][tx][0] = make_float4(sk[0], sk[1], sk[2], sk[3]);
            part_s[b][warp][tx][1] = make_float4(sq[0], sq[1], sq[2], sq[3]);
        }
        if (i + 1 < s.count) stage(i + 1);
        __syncthreads();
        float4 ak = make_float4(0.f, 0.f, 0.f, 0.f), aq = ak;
#pragma unroll
        for (int w = 0; w < RC_WARPS; ++w) {
            if constexpr (DELTA) { const float4 t = part_s[b][w][tx][0]; ak.x += t.x; ak.y += t.y; ak.z += t.z; ak.w += t.w; }
            const float4 t = part_s[b][w][tx][1];
            aq.x += t.x; aq.y += t.y; aq.z += t.z; aq.w += t.w;
        }
        const float a4[4] = {ak.x, ak.y, ak.z, ak.w}, r4[4] = {aq.x, aq.y, aq.z, aq.w};
        float u[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) u[e] = DELTA ? beta * (v[e] - a4[e] * kn) : MODE == 3 ? g_s[c][1] * v[e] : v[e];
        if (ty == 0)
            for (int e = 0; e < live; ++e) P.out[r * P.H * Dv + (size_t)h * Dv + col + e] = qn * (r4[e] + qk * kn * u[e]) + (MODE == 3 ? skip * v[e] : 0.f);
#pragma unroll
        for (int j = 0; j < RM; ++j) {
            const float k = k_s[c][ty + 32 * j] * kn;
#pragma unroll
            for (int e = 0; e < 4; ++e) S[j][e] = fmaf(k, u[e], S[j][e]);
        }
    }
#pragma unroll
    for (int i = 0; i < RM; ++i) {
        const int d = ty + 32 * i;
        if (d < D && live > 0) {
            if (vec) *reinterpret_cast<float4*>(st + (size_t)d * Dv + col) = make_float4(S[i][0], S[i][1], S[i][2], S[i][3]);
            else
                for (int e = 0; e < live; ++e) st[(size_t)d * Dv + col + e] = S[i][e];
        }
    }
}

// ---------------------------------------------------------------------------------------------- norm and gate
// TPG threads per group of gs columns; with V = 4, gs and every pitch are multiples of four.
template <typename T, typename TG, int TPG, int V>
__global__ void __launch_bounds__(256) group_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ w, const TG* __restrict__ gate,
                                                              long long ld_gate, T* __restrict__ out, long long groups, int per_row, int gs, float eps, int act, int first,
                                                              int w_row) {
    __shared__ float red[8];
    pdl_wait();
    pdl_launch_dependents();
    const long long grp = (long long)blockIdx.x * (256 / TPG) + threadIdx.x / TPG;
    const int t = threadIdx.x % TPG;
    if (grp >= groups) return;                         // whole warps; with 256 threads per group the whole CTA
    const long long row = grp / per_row;
    const int at = (int)(grp % per_row) * gs;
    const float* src = o + row * per_row * gs + at;
    const TG* gp = gate + row * ld_gate + at;
    const float* wp = w + (w_row ? at : 0);
    float ss = 0.f;
    for (int c = t * V; c < gs; c += TPG * V) {
        Elems<float, V> f = ld_elems<float, V>(src + c);
        if (first) {
            const Elems<TG, V> g = ld_elems<TG, V>(gp + c);
#pragma unroll
            for (int e = 0; e < V; ++e) f.v[e] *= act ? silu(g.v[e]) : sigmoid(g.v[e]);
        }
#pragma unroll
        for (int e = 0; e < V; ++e) ss += f.v[e] * f.v[e];
    }
    ss = warp_sum(ss);
    if constexpr (TPG == 256) {
        if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int i = 0; i < 8; ++i) ss += red[i];
    }
    const float rs = rsqrtf(ss / (float)gs + eps);
    T* op = out + row * per_row * gs + at;
    for (int c = t * V; c < gs; c += TPG * V) {
        const Elems<float, V> f = ld_elems<float, V>(src + c), m = ld_elems<float, V>(wp + c);
        const Elems<TG, V> g = ld_elems<TG, V>(gp + c);
        Elems<T, V> r;
#pragma unroll
        for (int e = 0; e < V; ++e) r.v[e] = f.v[e] * rs * m.v[e] * (act ? silu(g.v[e]) : sigmoid(g.v[e]));
        st_elems<T, V>(op + c, r);
    }
}

template <typename T, typename TG>
static cudaError_t norm_gate_launch(const float* o, const float* w, const void* gate, long long ld_gate, void* out, long long n, int per_row, int gs,
                                    float eps, int act, int first, int w_row, bool vec, cudaStream_t st) {
    const long long groups = n * per_row;
    auto go = [&](auto k, int tpg) {
        return ptb_launch(k, dim3((unsigned)((groups + 256 / tpg - 1) / (256 / tpg))), dim3(256), 0, st, ptb_pdl_enabled(), o, w, (const TG*)gate, ld_gate,
                          (T*)out, groups, per_row, gs, eps, act, first, w_row);
    };
    if (gs > 512) return vec ? go(group_norm_gate_kernel<T, TG, 256, 4>, 256) : go(group_norm_gate_kernel<T, TG, 256, 1>, 256);
    return vec ? go(group_norm_gate_kernel<T, TG, 32, 4>, 32) : go(group_norm_gate_kernel<T, TG, 32, 1>, 32);
}

template <typename T, int MODE>
static cudaError_t recurrence_launch(const PtbRecurrence& p, cudaStream_t st) {
    const dim3 grid((p.Dv + RC_COLS - 1) / RC_COLS, p.H, p.seqs ? p.n_seqs : p.n);
    auto go = [&](auto k) { return ptb_launch(k, grid, dim3(RC_THREADS), 0, st, ptb_pdl_enabled(), p); };
    if (p.D <= 32) return go(recurrence_kernel<T, MODE, 1>);
    if (p.D <= 64) return go(recurrence_kernel<T, MODE, 2>);
    if (p.D <= 128) return go(recurrence_kernel<T, MODE, 4>);
    if (p.D <= 256) return go(recurrence_kernel<T, MODE, 8>);
    return go(recurrence_kernel<T, MODE, 16>);
}

int recurrence_check(const PtbRecurrence& p) {
    if (p.H < 1 || p.G < 1 || p.H % p.G || p.D < 1 || p.D > 512 || p.Dv < 1 || p.H > 65535) {
        ptb_set_error("recurrence: bad sizes (H %d, G %d, D %d, Dv %d; D at most 512)", p.H, p.G, p.D, p.Dv);
        return -1;
    }
    if (!p.x || !p.state || !p.out || !p.decay || (p.delta && ((!p.a && !p.low) || (p.delta == 3 ? !p.skip : !p.beta) || !p.dt_bias))) { ptb_set_error("recurrence: missing operand"); return -1; }
    if ((p.seqs ? p.n_seqs : p.n) > 65535) { ptb_set_error("recurrence: more than 65535 sequences in one launch"); return -1; }
    return 0;
}

}  // namespace ptb

using namespace ptb;

// out [n, C] = silu(causal convolution of x [n, C] (pitch ld) + bias) with w [taps][C] and bias [C] (or null) fp32, the current token's tap last; `add`:
// out = x + the convolution + bias.  state [slots][taps - 1][C] in the type of x.  seqs [n_seqs] int4 (first row, rows, first position, slot): a prompt pass; null: one token per row.
PTB_API int ptb_short_conv(const void* x, long long ld, const float* w, const float* bias, int add, int C, int taps, void* state, void* out, int n, int slots, const int* pos,
                           int pos_stride, const int* req, int req_stride, const void* seqs, int n_seqs, int* status, int bf16, cudaStream_t st) {
    if (n <= 0 || C <= 0) return 0;
    if (taps < 1 || slots < 1 || n_seqs > 65535) { ptb_set_error("short_conv: %d taps, %d slots, %d sequences", taps, slots, n_seqs); return -1; }
    const int per = seqs ? CONV_TOKENS : 1;
    const long long rows = ((long long)n + per - 1) / per;
    if (rows > 65535) { ptb_set_error("short_conv: %d rows in one launch", n); return -1; }
    ConvParams p{x, ld, w, bias, add, state, out, pos, req, (const int4*)seqs, C, taps, n, slots, pos_stride, req_stride, n_seqs, status};
    const bool vec = C % 8 == 0 && ld % 8 == 0 && (((uintptr_t)x | (uintptr_t)w | (uintptr_t)bias | (uintptr_t)state | (uintptr_t)out) & 15) == 0;
    const int lanes = vec ? C / 8 : C, threads = lanes >= 256 ? 256 : (lanes + 31) / 32 * 32;
    const dim3 grid((lanes + threads - 1) / threads, (unsigned)rows);
    const bool pdl = ptb_pdl_enabled();
    if (bf16 && vec && seqs && taps >= 2 && taps <= 4)
        PTB_CUDA_OK(ptb_launch(taps == 2 ? short_conv_taps_kernel<__nv_bfloat16, 8, 2> : taps == 3 ? short_conv_taps_kernel<__nv_bfloat16, 8, 3> : short_conv_taps_kernel<__nv_bfloat16, 8, 4>,
                               grid, dim3(threads), 0, st, pdl, p));
    else if (bf16) PTB_CUDA_OK(ptb_launch(vec ? short_conv_kernel<__nv_bfloat16, 8> : short_conv_kernel<__nv_bfloat16, 1>, grid, dim3(threads), 0, st, pdl, p));
    else PTB_CUDA_OK(ptb_launch(vec ? short_conv_kernel<float, 8> : short_conv_kernel<float, 1>, grid, dim3(threads), 0, st, pdl, p));
    if (seqs && taps > 1) {
        const dim3 tail((C + 255) / 256, n_seqs);
        if (bf16) PTB_CUDA_OK(ptb_launch(conv_tail_kernel<__nv_bfloat16>, tail, dim3(256), 0, st, pdl, p));
        else PTB_CUDA_OK(ptb_launch(conv_tail_kernel<float>, tail, dim3(256), 0, st, pdl, p));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// A recurrent layer over the rows of a batch, token by token; see PtbRecurrence.
PTB_API int ptb_recurrence(const PtbRecurrence* args, cudaStream_t st) {
    const PtbRecurrence& p = *args;
    if (p.n <= 0 || (p.seqs && p.n_seqs <= 0)) return 0;
    if (recurrence_check(p)) return -1;
    if (p.delta && !p.a) { ptb_set_error("recurrence: token by token takes a, not its low-rank factors"); return -1; }
    if (p.delta < 0 || p.delta > 3) { ptb_set_error("recurrence: kind %d", p.delta); return -1; }
    auto go = p.bf16 ? (p.delta == 3 ? recurrence_launch<__nv_bfloat16, 3> : p.delta == 2 ? recurrence_launch<__nv_bfloat16, 2> : p.delta ? recurrence_launch<__nv_bfloat16, 1> : recurrence_launch<__nv_bfloat16, 0>)
                     : (p.delta == 3 ? recurrence_launch<float, 3> : p.delta == 2 ? recurrence_launch<float, 2> : p.delta ? recurrence_launch<float, 1> : recurrence_launch<float, 0>);
    PTB_CUDA_OK(go(p, st));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out [n, per_row gs] (bf16 or fp32) = o / rms(o) * w * act(gate), act the sigmoid (0) or SiLU (1), o fp32 in groups of gs columns, w [gs] fp32, gate [n, per_row gs] with
// row pitch ld_gate in bf16 (gate_bf16) or fp32.  first: out = g / rms(g) * w with g = o act(gate) instead; w_row: w is [per_row gs].
PTB_API int ptb_group_norm_gate(const float* o, const float* w, const void* gate, int gate_bf16, long long ld_gate, void* out, int n, int per_row,
                                int gs, float eps, int act, int first, int w_row, int bf16, cudaStream_t st) {
    if (n <= 0 || per_row <= 0 || gs <= 0) return 0;
    const bool vec = gs % 4 == 0 && ld_gate % 4 == 0 && (((uintptr_t)o | (uintptr_t)w | (uintptr_t)out | (uintptr_t)gate) & 15) == 0;
    cudaError_t e;
    if (bf16) e = gate_bf16 ? norm_gate_launch<__nv_bfloat16, __nv_bfloat16>(o, w, gate, ld_gate, out, n, per_row, gs, eps, act, first, w_row, vec, st)
                            : norm_gate_launch<__nv_bfloat16, float>(o, w, gate, ld_gate, out, n, per_row, gs, eps, act, first, w_row, vec, st);
    else e = gate_bf16 ? norm_gate_launch<float, __nv_bfloat16>(o, w, gate, ld_gate, out, n, per_row, gs, eps, act, first, w_row, vec, st)
                       : norm_gate_launch<float, float>(o, w, gate, ld_gate, out, n, per_row, gs, eps, act, first, w_row, vec, st);
    PTB_CUDA_OK(e);
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
