// Decode-side kernels of gated attention (gated_attn.cuh):
//   head_norm_write_kernel    after the packed q/k/v projection: RMS norm of every q and k head, value mixing, page write;
//   gated_rows_mma_kernel     bf16, one CTA per (query row, split of its window), all heads: the head mixing couples them.
//                             Tensor-core products straight from the pages, scores and weights in fp32;
//   gated_rows_f32_kernel     the same in true fp32 arithmetic (FMA);
//   gated_merge_kernel        sums the splits.
// Page ids, positions and page-table columns are checked against their extents; a bad one sets PTB_ERR_BOUNDS and its key counts
// as invisible.
#include "gated_attn.cuh"
#include "flash_attn.cuh"
#include <algorithm>

namespace ptb {

constexpr int GA_THREADS = 256;
constexpr int GA_WARPS = GA_THREADS / 32;

// ---------------------------------------------------------------------------------------------- norm + page write
struct HeadNormParams {
    const void* qkv;                   // [n] rows: q heads, k heads from k_col on, v heads from v_col on
    long long ld;
    int k_col, v_col;
    void* q_out;                       // [n, H, Dp], the pad filled with zeros
    void* k_pages;
    void* v_pages;
    const float* qw;                   // [D] or null
    const float* kw;                   // [D] or null
    const float* gain;                 // [positions]: q times the entry of its position; or null
    int positions;
    const void* v_first;               // rows of another layer's values [n, G Dv] (pitch v_first_ld), or null
    long long v_first_ld;
    float lam;                         // v = (1 - lam) v + lam v_first
    const int* pos;
    const int* req;
    const int* page_table;
    int pos_stride, req_stride, pt_stride, n_pages;
    int H, G, D, Dp, Dv, Dvp;
    float eps;
    int* status;
};

template <typename T> struct Vec8T;
template <> struct Vec8T<__nv_bfloat16> {
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float* f) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 v = __bfloat1622float2(h[i]); f[2 * i] = v.x; f[2 * i + 1] = v.y; }
    }
    static __device__ __forceinline__ void store(__nv_bfloat16* p, const float* f) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    }
};
template <> struct Vec8T<float> {
    static __device__ __forceinline__ void load(const float* p, float* f) {
        const float4 a = reinterpret_cast<const float4*>(p)[0], b = reinterpret_cast<const float4*>(p)[1];
        f[0] = a.x; f[1] = a.y; f[2] = a.z; f[3] = a.w; f[4] = b.x; f[5] = b.y; f[6] = b.z; f[7] = b.w;
    }
    static __device__ __forceinline__ void store(float* p, const float* f) {
        reinterpret_cast<float4*>(p)[0] = make_float4(f[0], f[1], f[2], f[3]);
        reinterpret_cast<float4*>(p)[1] = make_float4(f[4], f[5], f[6], f[7]);
    }
};
__device__ __forceinline__ float ga_f(float v) { return v; }
__device__ __forceinline__ float ga_f(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T ga_t(float v);
template <> __device__ __forceinline__ float ga_t<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 ga_t<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// `lph` lanes share a head (a power of two); E = elements a lane handles per step (8: vector access, 1: any size).
template <typename T, int E>
__global__ void __launch_bounds__(256) head_norm_write_kernel(const __grid_constant__ HeadNormParams P, int lph) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = blockIdx.x;
    const int pos = P.pos[i * P.pos_stride], col = pos / GA_PAGE, slot = pos % GA_PAGE;
    int page = -1;
    if (pos >= 0 && col < P.pt_stride) page = P.page_table[(size_t)P.req[i * P.req_stride] * P.pt_stride + col];
    if (page < 0 || page >= P.n_pages) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        page = -1;
    }
    float factor = 1.f;
    if (P.gain) {
        if ((pos < 0 || pos >= P.positions) && threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        factor = P.gain[min(max(pos, 0), P.positions - 1)];
    }
    const T* row = (const T*)P.qkv + i * P.ld;
    const int sub = threadIdx.x % lph, group = threadIdx.x / lph, groups = blockDim.x / lph;
    const int heads = P.H + 2 * P.G;
    // whole groups stay in the loop together (a warp's groups may differ in their last round, so the shuffles name their lanes)
    const unsigned mask = lph == 32 ? 0xffffffffu : ((1u << lph) - 1u) << ((threadIdx.x & 31) / lph * lph);
    for (int h = group; h < heads; h += groups) {
        const bool is_q = h < P.H, is_v = h >= P.H + P.G;
        const int width = is_v ? P.Dv : P.D, padded = is_v ? P.Dvp : P.Dp;
        const T* src = row + (is_v ? P.v_col + (size_t)(h - P.H - P.G) * P.Dv : is_q ? (size_t)h * P.D : P.k_col + (size_t)(h - P.H) * P.D);
        T* dst;
        if (is_q) dst = (T*)P.q_out + (i * P.H + h) * P.Dp;
        else {
            if (page < 0) continue;
            const int g = is_v ? h - P.H - P.G : h - P.H;
            dst = (is_v ? (T*)P.v_pages : (T*)P.k_pages) + (((size_t)page * P.G + g) * GA_PAGE + slot) * padded;
        }
        float rs = 1.f;
        if (!is_v) {
            float ss = 0.f;
            for (int c = sub * E; c < width; c += lph * E) {
                if constexpr (E == 8) {
                    float f[8];
                    Vec8T<T>::load(src + c, f);
#pragma unroll
                    for (int e = 0; e < 8; ++e) ss += f[e] * f[e];
                } else {
                    const float f = ga_f(src[c]);
                    ss += f * f;
                }
            }
            for (int o = lph / 2; o > 0; o >>= 1) ss += __shfl_xor_sync(mask, ss, o);
            rs = rsqrtf(ss / (float)width + P.eps);
            if (is_q) rs *= factor;
        }
        const float* w = is_q ? P.qw : P.kw;
        const T* vf = is_v && P.v_first ? (const T*)P.v_first + i * P.v_first_ld + (size_t)(h - P.H - P.G) * P.Dv : nullptr;
        for (int c = sub * E; c < padded; c += lph * E) {
            if constexpr (E == 8) {
                float f[8];
                if (c < width) {
                    Vec8T<T>::load(src + c, f);
                    if (!is_v) {
#pragma unroll
                        for (int e = 0; e < 8; ++e) f[e] = f[e] * rs * (w ? w[c + e] : 1.f);
                    } else if (vf) {
                        float g[8];
                        Vec8T<T>::load(vf + c, g);
#pragma unroll
                        for (int e = 0; e < 8; ++e) f[e] = (1.f - P.lam) * f[e] + P.lam * g[e];
                    }
                } else {
#pragma unroll
                    for (int e = 0; e < 8; ++e) f[e] = 0.f;
                }
                Vec8T<T>::store(dst + c, f);
            } else {
                float f = 0.f;
                if (c < width) {
                    f = ga_f(src[c]);
                    if (!is_v) f = f * rs * (w ? w[c] : 1.f);
                    else if (vf) f = (1.f - P.lam) * f + P.lam * ga_f(vf[c]);
                }
                dst[c] = ga_t<T>(f);
            }
        }
    }
}

// ---------------------------------------------------------------------------------------------- one query row
// The keys of split `split` of row `i`: [j0, j0 + nk), their cache slots (page * 64 + slot, or -1) in krow.
struct RowSpan { int pos, j0, nk; };
__device__ __forceinline__ RowSpan row_span(const GatedAttnParams& P, int i, int split, int* krow, int kpad) {
    RowSpan r;
    r.pos = P.pos[(size_t)i * P.pos_stride];
    const int lo = max(0, r.pos - P.window + 1), cnt = max(0, r.pos - lo + 1);
    int kps = (cnt + P.nsplit - 1) / P.nsplit;
    if (r.pos < 0 || kps > P.kcap) {                   // the host sizes the splits for the longest row
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        kps = min(kps, P.kcap);
    }
    r.j0 = lo + split * kps;
    r.nk = max(0, min(kps, r.pos + 1 - r.j0));
    const int* table = P.page_table + (size_t)P.req[(size_t)i * P.req_stride] * P.pt_stride;
    for (int e = threadIdx.x; e < kpad; e += blockDim.x) {
        int v = -1;
        if (e < r.nk) {
            const int j = r.j0 + e, col = j / GA_PAGE;
            const int page = col < P.pt_stride ? table[col] : -1;
            if (page >= 0 && page < P.n_pages) v = page * GA_PAGE + j % GA_PAGE;
            else if (P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        }
        krow[e] = v;
    }
    return r;
}
__device__ __forceinline__ size_t kv_row(int krow, int G, int g) { return ((size_t)(krow / GA_PAGE) * G + g) * GA_PAGE + krow % GA_PAGE; }

struct RowSmem {
    int q, w, hi, lo, talk, krow, total;               // byte offsets
    __host__ __device__ RowSmem(int H, int Dp, int kcap, int elt) {
        q = 0;
        w = q + H * Dp * elt;
        hi = w + H * (kcap + 1) * 4;
        hi = (hi + 15) & ~15;
        lo = hi + (elt == 2 ? H * (kcap + 8) * 2 : H * (kcap + 1) * 4);
        talk = lo + (elt == 2 ? H * (kcap + 8) * 2 : 0);
        talk = (talk + 15) & ~15;
        krow = talk + H * ((H + 3) & ~3) * 4;
        total = krow + kcap * 4;
    }
};

// Head mixing of the weights of `kpad` keys: calls put(h, key, value) for every head and key.
template <typename F>
__device__ __forceinline__ void mix_heads(const float* w_s, const float* talk_s, int H, int ldw, int kpad, bool talk, F put) {
    const int H4 = (H + 3) / 4, ldt = H4 * 4;
    for (int e = threadIdx.x; e < H4 * kpad; e += blockDim.x) {
        const int hq = e / kpad, j = e % kpad;
        float a[4] = {0.f, 0.f, 0.f, 0.f};
        if (talk) {
            for (int g = 0; g < H; ++g) {
                const float wv = w_s[g * ldw + j];
                const float4 t = *reinterpret_cast<const float4*>(talk_s + g * ldt + hq * 4);
                a[0] = fmaf(t.x, wv, a[0]); a[1] = fmaf(t.y, wv, a[1]); a[2] = fmaf(t.z, wv, a[2]); a[3] = fmaf(t.w, wv, a[3]);
            }
        } else {
#pragma unroll
            for (int k = 0; k < 4; ++k) if (hq * 4 + k < H) a[k] = w_s[(hq * 4 + k) * ldw + j];
        }
#pragma unroll
        for (int k = 0; k < 4; ++k) if (hq * 4 + k < H) put(hq * 4 + k, j, a[k]);
    }
}
__device__ __forceinline__ void load_talk(const GatedAttnParams& P, float* talk_s) {     // transposed: [from][to, padded to 4]
    if (!P.talk) return;
    const int ldt = (P.H + 3) & ~3;
    for (int e = threadIdx.x; e < P.H * ldt; e += blockDim.x) {
        const int f = e / ldt, h = e % ldt;
        talk_s[e] = h < P.H ? P.talk[(size_t)h * P.H + f] : 0.f;
    }
}

// A lane of a quad (g = lane / 4, t = lane % 4) loads 16 bytes = 8 consecutive elements of a key's vector and uses them as its
// elements of two k16 steps; the query's fragment takes the same elements, so the order inside a 32-element group cancels.
__global__ void __launch_bounds__(GA_THREADS) gated_rows_mma_kernel(const __grid_constant__ GatedAttnParams P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const RowSmem L(P.H, P.Dp, P.kcap, 2);
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem + L.q);
    float* w_s = reinterpret_cast<float*>(smem + L.w);
    __nv_bfloat16* hi_s = reinterpret_cast<__nv_bfloat16*>(smem + L.hi);
    __nv_bfloat16* lo_s = reinterpret_cast<__nv_bfloat16*>(smem + L.lo);
    float* talk_s = reinterpret_cast<float*>(smem + L.talk);
    int* krow = reinterpret_cast<int*>(smem + L.krow);
    const int split = blockIdx.x, i = blockIdx.y, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int ldw = P.kcap + 1, ldh = P.kcap + 8, R = P.H / P.G, RB = (R + 7) / 8;
    load_talk(P, talk_s);                              // constant over the run: not written by the kernel before
    pdl_wait();
    pdl_launch_dependents();
    const RowSpan S = row_span(P, i, split, krow, P.kcap);
    {
        const uint4* src = reinterpret_cast<const uint4*>((const __nv_bfloat16*)P.q + (size_t)i * P.H * P.Dp);
        uint4* dst = reinterpret_cast<uint4*>(q_s);
        for (int e = threadIdx.x; e < P.H * P.Dp / 8; e += GA_THREADS) dst[e] = src[e];
    }
    __syncthreads();
    const int kgroups = (S.nk + 15) / 16, kpad = kgroups * 16;
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    const __nv_bfloat16* kp = (const __nv_bfloat16*)P.k_pages;
    for (int u = warp; u < P.G * RB * kgroups; u += GA_WARPS) {
        const int kg = u % kgroups, rb = (u / kgroups) % RB, c = u / (kgroups * RB);
        const int r0 = krow[kg * 16 + g], r1 = krow[kg * 16 + g + 8];
        const uint4* k0 = reinterpret_cast<const uint4*>(kp + kv_row(max(r0, 0), P.G, c) * P.Dp);
        const uint4* k1 = reinterpret_cast<const uint4*>(kp + kv_row(max(r1, 0), P.G, c) * P.Dp);
        const int head = c * R + rb * 8 + g;           // this lane's column of the query fragment
        const bool head_ok = rb * 8 + g < R;
        const uint4* qv = reinterpret_cast<const uint4*>(q_s + (size_t)(head_ok ? head : 0) * P.Dp);
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
        const int nch = P.Dp / 8;
        for (int b0 = 0; b0 < nch; b0 += 16) {
            uint4 a[4], b[4];
#pragma unroll
            for (int s = 0; s < 4; ++s) {
                const int ch = b0 + s * 4 + t;
                a[s] = (ch < nch && r0 >= 0) ? k0[ch] : zero4;
                b[s] = (ch < nch && r1 >= 0) ? k1[ch] : zero4;
            }
#pragma unroll
            for (int s = 0; s < 4; ++s) {
                const int ch = b0 + s * 4 + t;
                if (b0 + s * 4 < nch) {
                    const uint4 q4 = (ch < nch && head_ok) ? qv[ch] : zero4;
                    const uint32_t f0[4] = {a[s].x, b[s].x, a[s].y, b[s].y}, f1[4] = {a[s].z, b[s].z, a[s].w, b[s].w};
                    fa::mma16816(acc, f0, q4.x, q4.y);
                    fa::mma16816(acc, f1, q4.z, q4.w);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int key = kg * 16 + g + (e >> 1) * 8, hl = rb * 8 + 2 * t + (e & 1);
            if (hl < R) {
                const int h = c * R + hl;
                const bool ok = ((e >> 1) ? r1 : r0) >= 0;
                w_s[h * ldw + key] = ok ? gated_weight(P, acc[e], h, S.pos - S.j0 - key) : 0.f;
            }
        }
    }
    __syncthreads();
    mix_heads(w_s, talk_s, P.H, ldw, kpad, P.talk != nullptr, [&](int h, int j, float v) {
        const __nv_bfloat16 hi = __float2bfloat16_rn(v);
        hi_s[h * ldh + j] = hi;
        lo_s[h * ldh + j] = __float2bfloat16_rn(v - __bfloat162float(hi));
    });
    __syncthreads();
    // o^T tile: rows 0-7 of the MMA carry the high halves of eight heads' weights, rows 8-15 the low halves; columns are values.
    // Lane (g, t) loads 16 bytes at value chunk g of the keys 2t, 2t+1, 2t+8, 2t+9: element e of the chunk is its column of tile e.
    const __nv_bfloat16* vp = (const __nv_bfloat16*)P.v_pages;
    const int DC = (P.Dvp + 63) / 64;
    for (int u = warp; u < P.G * RB * DC; u += GA_WARPS) {
        const int dc = u % DC, rb = (u / DC) % RB, c = u / (DC * RB);
        const int h = c * R + rb * 8 + g;
        const bool head_ok = rb * 8 + g < R, ch_ok = dc * 64 + g * 8 < P.Dvp;
        const __nv_bfloat16* hi_r = hi_s + (head_ok ? h : 0) * ldh + 2 * t;
        const __nv_bfloat16* lo_r = lo_s + (head_ok ? h : 0) * ldh + 2 * t;
        float acc[8][4];
#pragma unroll
        for (int e = 0; e < 8; ++e)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[e][k] = 0.f;
#pragma unroll 2
        for (int kg = 0; kg < kgroups; ++kg) {
            uint4 v[4];
#pragma unroll
            for (int k = 0; k < 4; ++k) {
                const int r = krow[kg * 16 + 2 * t + (k & 1) + (k >> 1) * 8];
                v[k] = (r >= 0 && ch_ok) ? *reinterpret_cast<const uint4*>(vp + kv_row(r, P.G, c) * P.Dvp + dc * 64 + g * 8) : zero4;
            }
            uint32_t a[4] = {0u, 0u, 0u, 0u};
            if (head_ok) {
                a[0] = *reinterpret_cast<const uint32_t*>(hi_r + kg * 16);
                a[1] = *reinterpret_cast<const uint32_t*>(lo_r + kg * 16);
                a[2] = *reinterpret_cast<const uint32_t*>(hi_r + kg * 16 + 8);
                a[3] = *reinterpret_cast<const uint32_t*>(lo_r + kg * 16 + 8);
            }
            const uint32_t* w0 = reinterpret_cast<const uint32_t*>(&v[0]);
            const uint32_t* w1 = reinterpret_cast<const uint32_t*>(&v[1]);
            const uint32_t* w2 = reinterpret_cast<const uint32_t*>(&v[2]);
            const uint32_t* w3 = reinterpret_cast<const uint32_t*>(&v[3]);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                fa::mma16816(acc[2 * e], a, __byte_perm(w0[e], w1[e], 0x5410), __byte_perm(w2[e], w3[e], 0x5410));
                fa::mma16816(acc[2 * e + 1], a, __byte_perm(w0[e], w1[e], 0x7632), __byte_perm(w2[e], w3[e], 0x7632));
            }
        }
        if (!head_ok) continue;
        // columns 2t and 2t+1 of tile e are the values dc*64 + 16t + e and dc*64 + 16t + 8 + e
        const int d0 = dc * 64 + 16 * t;
        if (P.nsplit > 1) {
            if (d0 < P.Dvp) {                          // Dvp is a multiple of 16
                float4* o = reinterpret_cast<float4*>(P.work + (((size_t)i * P.nsplit + split) * P.H + h) * P.Dvp + d0);
#pragma unroll
                for (int s = 0; s < 2; ++s)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        o[s * 2 + e] = make_float4(acc[4 * e][s] + acc[4 * e][s + 2], acc[4 * e + 1][s] + acc[4 * e + 1][s + 2],
                                                   acc[4 * e + 2][s] + acc[4 * e + 2][s + 2], acc[4 * e + 3][s] + acc[4 * e + 3][s + 2]);
            }
        } else {
            __nv_bfloat16* o = (__nv_bfloat16*)P.out + (size_t)i * P.H * P.Dv + (size_t)h * P.Dv;
#pragma unroll
            for (int s = 0; s < 2; ++s)
#pragma unroll
                for (int e = 0; e < 8; ++e)
                    if (d0 + s * 8 + e < P.Dv) o[d0 + s * 8 + e] = __float2bfloat16_rn(acc[e][s] + acc[e][s + 2]);
        }
    }
}

__global__ void __launch_bounds__(GA_THREADS) gated_rows_f32_kernel(const __grid_constant__ GatedAttnParams P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const RowSmem L(P.H, P.Dp, P.kcap, 4);
    float* q_s = reinterpret_cast<float*>(smem + L.q);
    float* w_s = reinterpret_cast<float*>(smem + L.w);
    float* m_s = reinterpret_cast<float*>(smem + L.hi);
    float* talk_s = reinterpret_cast<float*>(smem + L.talk);
    int* krow = reinterpret_cast<int*>(smem + L.krow);
    const int split = blockIdx.x, i = blockIdx.y, ldw = P.kcap + 1, R = P.H / P.G;
    load_talk(P, talk_s);
    pdl_wait();
    pdl_launch_dependents();
    const RowSpan S = row_span(P, i, split, krow, P.kcap);
    for (int e = threadIdx.x; e < P.H * P.Dp; e += GA_THREADS) q_s[e] = ((const float*)P.q)[(size_t)i * P.H * P.Dp + e];
    __syncthreads();
    for (int e = threadIdx.x; e < P.H * S.nk; e += GA_THREADS) {
        const int h = e / S.nk, j = e % S.nk, r = krow[j];
        float w = 0.f;
        if (r >= 0) {
            const float4* k4 = reinterpret_cast<const float4*>((const float*)P.k_pages + kv_row(r, P.G, h / R) * P.Dp);
            const float4* q4 = reinterpret_cast<const float4*>(q_s + (size_t)h * P.Dp);
            float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int d = 0; d < P.Dp / 4; ++d) {
                const float4 a = k4[d], b = q4[d];
                s.x = fmaf(a.x, b.x, s.x); s.y = fmaf(a.y, b.y, s.y); s.z = fmaf(a.z, b.z, s.z); s.w = fmaf(a.w, b.w, s.w);
            }
            w = gated_weight(P, (s.x + s.y) + (s.z + s.w), h, S.pos - S.j0 - j);
        }
        w_s[h * ldw + j] = w;
    }
    __syncthreads();
    if (S.nk > 0)
        mix_heads(w_s, talk_s, P.H, ldw, S.nk, P.talk != nullptr, [&](int h, int j, float v) { m_s[h * ldw + j] = v; });
    __syncthreads();
    for (int e = threadIdx.x; e < P.H * P.Dvp; e += GA_THREADS) {
        const int h = e / P.Dvp, d = e % P.Dvp;
        float a = 0.f;
        for (int j = 0; j < S.nk; ++j)
            if (krow[j] >= 0) a = fmaf(m_s[h * ldw + j], ((const float*)P.v_pages)[kv_row(krow[j], P.G, h / R) * P.Dvp + d], a);
        if (P.nsplit > 1) P.work[(((size_t)i * P.nsplit + split) * P.H + h) * P.Dvp + d] = a;
        else if (d < P.Dv) ((float*)P.out)[((size_t)i * P.H + h) * P.Dv + d] = a;
    }
}

// out [n, H * Dv] = sum over the splits; a thread sums four neighbouring values.
template <typename T>
__global__ void __launch_bounds__(256) gated_merge_kernel(const float* __restrict__ work, T* __restrict__ out, int H, int Dv, int Dvp, int nsplit) {
    pdl_wait();
    pdl_launch_dependents();
    const int q = blockIdx.x * blockDim.x + threadIdx.x, per = H * Dvp / 4;
    if (q >= per) return;
    const size_t i = blockIdx.y;
    const float4* w = reinterpret_cast<const float4*>(work + i * nsplit * (size_t)H * Dvp) + q;
    float4 a = w[0];
#pragma unroll 4
    for (int s = 1; s < nsplit; ++s) {
        const float4 v = w[(size_t)s * per];
        a.x += v.x; a.y += v.y; a.z += v.z; a.w += v.w;
    }
    const int h = q * 4 / Dvp, d = q * 4 % Dvp;
    T* o = out + i * H * (size_t)Dv + (size_t)h * Dv + d;
    if (d < Dv) o[0] = ga_t<T>(a.x);
    if (d + 1 < Dv) o[1] = ga_t<T>(a.y);
    if (d + 2 < Dv) o[2] = ga_t<T>(a.z);
    if (d + 3 < Dv) o[3] = ga_t<T>(a.w);
}

}  // namespace ptb

using namespace ptb;

// After the packed projection qkv (pitch ld; q heads first, k and v heads at k_col and v_col): q_out [n, H, Dp] = RMS norm of the q heads (weight qw
// [D]; null: none) times gain[pos] (fp32 [positions]; null: 1), the k heads' norm (kw) and the values go to the page slot of (req, pos).  v_first (pitch v_first_ld, optional) mixes another layer's
// values in: v = (1 - lam) v + lam v_first.  Dp, Dvp: sizes as stored, multiples of 16; the pad is zero.
PTB_API int ptb_head_norm_write(const void* qkv, long long ld, int k_col, int v_col, void* q_out, void* k_pages, void* v_pages, const float* qw, const float* kw,
                                const float* gain, int positions,
                                const void* v_first, long long v_first_ld, float lam, const int* pos, int pos_stride, const int* req,
                                int req_stride, const int* page_table, int pt_stride, int n_pages, int n, int H, int G, int D, int Dp,
                                int Dv, int Dvp, float eps, int* status, int bf16, cudaStream_t st) {
    if (n <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || Dp % 16 || Dvp % 16 || Dp < D || Dvp < Dv || (gain && positions < 1)) {
        ptb_set_error("head_norm_write: bad sizes (H %d, G %d, D %d/%d, Dv %d/%d)", H, G, D, Dp, Dv, Dvp);
        return -1;
    }
    HeadNormParams p;
    p.k_col = k_col; p.v_col = v_col; p.gain = gain; p.positions = positions;
    p.qkv = qkv; p.ld = ld; p.q_out = q_out; p.k_pages = k_pages; p.v_pages = v_pages; p.qw = qw; p.kw = kw; p.v_first = v_first;
    p.v_first_ld = v_first_ld; p.lam = lam; p.pos = pos; p.req = req; p.page_table = page_table; p.pos_stride = pos_stride;
    p.req_stride = req_stride; p.pt_stride = pt_stride; p.n_pages = n_pages; p.H = H; p.G = G; p.D = D; p.Dp = Dp; p.Dv = Dv; p.Dvp = Dvp;
    p.eps = eps; p.status = status;
    const int elt = bf16 ? 2 : 4;
    const bool vec = D % 8 == 0 && Dv % 8 == 0 && ld % 8 == 0 && (!v_first || v_first_ld % 8 == 0) && ((uintptr_t)qkv & 15) == 0 &&
                     ((uintptr_t)v_first & 15) == 0 && ((size_t)k_col * elt) % 16 == 0 && ((size_t)v_col * elt) % 16 == 0;
    const int steps = (std::max(Dp, Dvp) + (vec ? 7 : 0)) / (vec ? 8 : 1);
    int lph = 1;
    while (lph < steps && lph < 32) lph *= 2;
    const bool pdl = ptb_pdl_enabled();
    if (bf16) {
        auto k = vec ? head_norm_write_kernel<__nv_bfloat16, 8> : head_norm_write_kernel<__nv_bfloat16, 1>;
        PTB_CUDA_OK(ptb_launch(k, dim3(n), dim3(256), 0, st, pdl, p, lph));
    } else {
        auto k = vec ? head_norm_write_kernel<float, 8> : head_norm_write_kernel<float, 1>;
        PTB_CUDA_OK(ptb_launch(k, dim3(n), dim3(256), 0, st, pdl, p, lph));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// Floats of workspace the row kernels need for `nsplit` > 1.
PTB_API long long ptb_gated_rows_work_floats(int n, int H, int Dvp, int nsplit) { return nsplit > 1 ? (long long)n * nsplit * H * Dvp : 0; }

// Query rows q [n, H, Dp], each at its own position of its own sequence, against the cached keys inside their window.  max_keys: the
// most keys any row sees; nsplit CTAs share a row's keys (at most GA_KEYS each).  out [n, H Dv] in the type of q.
PTB_API int ptb_gated_attn_rows(const void* q, void* out, int n, int H, int G, int Dp, int Dv, int Dvp, const int* pos, int pos_stride,
                                const int* req, int req_stride, const int* page_table, int pt_stride, int n_pages, const void* k_pages,
                                const void* v_pages, const float* bias, int nb, const float* talk, int window, float scale, float cap,
                                int max_keys, float* work, int nsplit, int* status, int bf16, cudaStream_t st) {
    if (n <= 0) return 0;
    if (G <= 0 || H % G || Dp % 16 || Dvp % 16 || nb < 1 || window < 1) {
        ptb_set_error("gated attention: bad sizes (H %d, G %d, Dp %d, Dvp %d, nb %d, window %d)", H, G, Dp, Dvp, nb, window);
        return -1;
    }
    max_keys = std::max(1, std::min(max_keys, window));
    const int kps = (max_keys + nsplit - 1) / std::max(1, nsplit);
    if (nsplit < 1 || kps > GA_KEYS || (nsplit > 1 && !work)) {
        ptb_set_error("gated attention: %d splits for %d keys (at most %d keys per split, workspace needed above one)", nsplit, max_keys, GA_KEYS);
        return -1;
    }
    if (n > 65535) { ptb_set_error("gated attention: %d rows in one launch", n); return -1; }
    GatedAttnParams p;
    p.q = q; p.out = out; p.work = work; p.pos = pos; p.req = req; p.page_table = page_table; p.k_pages = k_pages; p.v_pages = v_pages;
    p.bias = bias; p.talk = talk; p.pos_stride = pos_stride; p.req_stride = req_stride; p.pt_stride = pt_stride; p.n_pages = n_pages;
    p.n = n; p.H = H; p.G = G; p.Dp = Dp; p.Dv = Dv; p.Dvp = Dvp; p.nb = nb; p.window = window; p.nsplit = nsplit;
    p.kcap = (kps + 15) & ~15; p.scale = scale; p.cap = cap; p.inv_cap = cap > 0.f ? 1.f / cap : 0.f; p.status = status;
    const RowSmem L(H, Dp, p.kcap, bf16 ? 2 : 4);
    if (L.total > 227 * 1024) { ptb_set_error("gated attention: %d heads of %d need %d bytes of shared memory", H, Dp, L.total); return -1; }
    auto kern = bf16 ? gated_rows_mma_kernel : gated_rows_f32_kernel;
    if (L.total > 48 * 1024) PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    const bool pdl = ptb_pdl_enabled();
    PTB_CUDA_OK(ptb_launch(kern, dim3(nsplit, n), dim3(GA_THREADS), (size_t)L.total, st, pdl, p));
    if (nsplit > 1) {
        const dim3 grid((H * Dvp / 4 + 255) / 256, n);
        if (bf16)
            PTB_CUDA_OK(ptb_launch(gated_merge_kernel<__nv_bfloat16>, grid, dim3(256), 0, st, pdl, (const float*)work, (__nv_bfloat16*)out, H, Dv, Dvp, nsplit));
        else
            PTB_CUDA_OK(ptb_launch(gated_merge_kernel<float>, grid, dim3(256), 0, st, pdl, (const float*)work, (float*)out, H, Dv, Dvp, nsplit));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
