// Row kernels of window attention (window_attn.cuh):
//   proj_norm_write_kernel   after the packed projection: RMS norm of the whole q and k rows, page write;
//   window_rows_mma_kernel   bf16, one CTA per (split of the keys, kv head, row).  Scores straight from the pages on the tensor cores,
//                            values on their way to shared memory meanwhile; a weight enters the value product as the sum of two
//                            bf16 numbers in the two halves of the 16-row operand;
//   window_rows_f32_kernel   the same in true fp32 arithmetic (FMA);
//   window_merge_kernel      joins the splits, the maps, the sink and the gate.
// With two maps the first half of a CTA's row blocks are the heads' first maps, the second half the second ones.
// Page ids, positions and page-table columns are checked against their extents; a bad one sets PTB_ERR_BOUNDS and its key counts
// as invisible.
#include "window_attn.cuh"
#include "flash_attn.cuh"
#include <algorithm>

namespace ptb {

template <typename T> __device__ __forceinline__ float wa_f(T v);
template <> __device__ __forceinline__ float wa_f<float>(float v) { return v; }
template <> __device__ __forceinline__ float wa_f<__nv_bfloat16>(__nv_bfloat16 v) { return __bfloat162float(v); }
template <typename T> __device__ __forceinline__ T wa_t(float v);
template <> __device__ __forceinline__ float wa_t<float>(float v) { return v; }
template <> __device__ __forceinline__ __nv_bfloat16 wa_t<__nv_bfloat16>(float v) { return __float2bfloat16_rn(v); }

// ---------------------------------------------------------------------------------------------- norm + page write
struct ProjNormParams {
    const void* x;
    long long ld;
    int q_col, k_col, v_col;
    void* q_out;                       // [n, H, Dp], the pad filled with zeros
    void* k_pages;
    void* v_pages;
    const float* qw;                   // [H D]
    const float* kw;                   // [G D]
    const int* pos;
    const int* req;
    const int* page_table;
    int pos_stride, req_stride, pt_stride, n_pages;
    int H, G, D, Dp, Dv, Dvp;
    float eps;
    int* status;
};

constexpr int PN_THREADS = 256;

// E elements per access: 8 where sizes and columns are multiples of eight, else 1.  One CTA per row.
template <typename T, int E>
__global__ void __launch_bounds__(PN_THREADS) proj_norm_write_kernel(const __grid_constant__ ProjNormParams P) {
    __shared__ float red[2][PN_THREADS / 32];
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = blockIdx.x;
    const int pos = P.pos[i * P.pos_stride], col = pos / WA_PAGE, slot = pos % WA_PAGE;
    int page = -1;
    if (pos >= 0 && col < P.pt_stride) page = P.page_table[(size_t)P.req[i * P.req_stride] * P.pt_stride + col];
    if (page < 0 || page >= P.n_pages) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        page = -1;
    }
    const T* row = (const T*)P.x + i * P.ld;
    struct Vec { float v[E]; };
    auto load = [&](const T* p) {
        Vec r;
        if constexpr (E == 8 && sizeof(T) == 2) {
            const uint4 raw = *reinterpret_cast<const uint4*>(p);
            const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
            for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h[e]); r.v[2 * e] = f.x; r.v[2 * e + 1] = f.y; }
        } else {
#pragma unroll
            for (int e = 0; e < E; ++e) r.v[e] = wa_f<T>(p[e]);
        }
        return r;
    };
    auto store = [&](T* p, const Vec& r) {
        if constexpr (E == 8 && sizeof(T) == 2) {
            uint4 raw;
            __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
            for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(r.v[2 * e], r.v[2 * e + 1]);
            *reinterpret_cast<uint4*>(p) = raw;
        } else {
#pragma unroll
            for (int e = 0; e < E; ++e) p[e] = wa_t<T>(r.v[e]);
        }
    };
    float sq = 0.f, sk = 0.f;
    for (int c = threadIdx.x * E; c < P.H * P.D; c += PN_THREADS * E) {
        const Vec f = load(row + P.q_col + c);
#pragma unroll
        for (int e = 0; e < E; ++e) sq += f.v[e] * f.v[e];
    }
    for (int c = threadIdx.x * E; c < P.G * P.D; c += PN_THREADS * E) {
        const Vec f = load(row + P.k_col + c);
#pragma unroll
        for (int e = 0; e < E; ++e) sk += f.v[e] * f.v[e];
    }
    sq = warp_sum(sq); sk = warp_sum(sk);
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sk; }
    __syncthreads();
    sq = sk = 0.f;
#pragma unroll
    for (int w = 0; w < PN_THREADS / 32; ++w) { sq += red[0][w]; sk += red[1][w]; }
    const float rq = rsqrtf(sq / (float)(P.H * P.D) + P.eps), rk = rsqrtf(sk / (float)(P.G * P.D) + P.eps);
    // heads of `width` columns from src to heads of `padded` elements `pitch` apart
    auto put = [&](const T* src, int heads, int width, int padded, T* dst, size_t pitch, const float* w, float rs) {
        for (int c = threadIdx.x * E; c < heads * padded; c += PN_THREADS * E) {
            const int h = c / padded, d = c % padded;
            Vec f;
#pragma unroll
            for (int e = 0; e < E; ++e) f.v[e] = 0.f;
            if (d < width) {
                f = load(src + h * width + d);
                if (w) {
#pragma unroll
                    for (int e = 0; e < E; ++e) f.v[e] *= rs * w[h * width + d + e];
                }
            }
            store(dst + h * pitch + d, f);
        }
    };
    put(row + P.q_col, P.H, P.D, P.Dp, (T*)P.q_out + i * P.H * P.Dp, P.Dp, P.qw, rq);
    if (page < 0) return;
    put(row + P.k_col, P.G, P.D, P.Dp, (T*)P.k_pages + ((size_t)page * P.G * WA_PAGE + slot) * P.Dp, (size_t)WA_PAGE * P.Dp, P.kw, rk);
    put(row + P.v_col, P.G, P.Dv, P.Dvp, (T*)P.v_pages + ((size_t)page * P.G * WA_PAGE + slot) * P.Dvp, (size_t)WA_PAGE * P.Dvp, nullptr, 1.f);
}

// ---------------------------------------------------------------------------------------------- one query row
struct WindowRows {
    PtbWindowAttn A;
    int kcap, hg, groups;              // keys of a CTA; query heads of a CTA, CTAs per kv head
    float scale_log2;                  // scale times log2(e)
};

// The cache slots (page * 64 + place, or -1) of the keys of split `split` of row `i`; returns their number and (dist) how the distance of the key
// at place e of the list follows from e.
struct Distance {
    int pos, e0, kept, lo;
    __device__ __forceinline__ int operator()(int e) const { return pos - (e0 + e < kept ? e0 + e : lo + e0 + e - kept); }
};
__device__ __forceinline__ int row_keys(const WindowRows& P, int i, int split, int* krow, Distance& dist) {
    const PtbWindowAttn& A = P.A;
    const int pos = A.pos[(size_t)i * A.pos_stride];
    const Seen s = seen_by(pos, A.window, A.keep, A.chunked);
    int per = (s.count + A.nsplit - 1) / A.nsplit;
    if (pos < 0 || per > P.kcap) {                     // the host sizes the splits for the row that sees most
        if (threadIdx.x == 0 && A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
        per = min(per, P.kcap);
    }
    const int e0 = split * per, nk = max(0, min(per, s.count - e0));
    dist = Distance{pos, e0, s.kept, s.lo};
    const int* table = A.page_table + (size_t)A.req[(size_t)i * A.req_stride] * A.pt_stride;
    for (int e = threadIdx.x; e < P.kcap; e += blockDim.x) {
        int v = -1;
        if (e < nk) {
            const int j = e0 + e < s.kept ? e0 + e : s.lo + e0 + e - s.kept, col = j / WA_PAGE;
            const int page = col < A.pt_stride ? table[col] : -1;
            if (page >= 0 && page < A.n_pages) v = page * WA_PAGE + j % WA_PAGE;
            else if (A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
        }
        krow[e] = v;
    }
    return nk;
}
__device__ __forceinline__ size_t cache_row(int krow, int G, int g) { return ((size_t)(krow / WA_PAGE) * G + g) * WA_PAGE + krow % WA_PAGE; }

// What a key's distance adds to a score of head h, in units of log2.
__device__ __forceinline__ float rel_log2(const PtbWindowAttn& A, int h, int distance) {
    return __ldg(A.rel + (size_t)h * A.rel_n + min(max(distance, 0), A.rel_n - 1)) * WA_LOG2E;
}

// Factor of a head's sum given its largest (log2) score and total: the sink joins the denominator, the gate multiplies.
template <typename T>
__device__ __forceinline__ float finish_factor(const PtbWindowAttn& A, size_t i, int h, float m, float l) {
    float M = m, f = 1.f;
    if (A.sink) {
        const float s = A.sink[h] * WA_LOG2E;
        M = fmaxf(m, s);
        f = m == -INFINITY ? 0.f : exp2f(m - M);
        l = l * f + exp2f(s - M);
    }
    f = l > 0.f ? f / l : 0.f;
    if (A.gate) f *= sigmoid(wa_f<T>(((const T*)A.gate)[i * A.gate_ld + h]));
    return f;
}

constexpr int WR_THREADS = 128, WR_WARPS = 4;

// The query heads of a CTA: `n` of them from h0, all of kv head c.
struct HeadGroup { int c, h0, n; };
__device__ __forceinline__ HeadGroup head_group(const WindowRows& P) {
    const int R = P.A.H / P.A.G, grp = blockIdx.y % P.groups;
    HeadGroup g;
    g.c = blockIdx.y / P.groups;
    g.h0 = g.c * R + grp * P.hg;
    g.n = min(P.hg, R - grp * P.hg);
    return g;
}

struct WindowSmem {
    int v, q, w, hi, lo, ml, krow, pitch, ldw, ldh, total;      // byte offsets; pitches in bytes (v) and elements
    __host__ __device__ WindowSmem(int rows, int Dp, int Dvp, int kcap, bool mma) {      // rows: of all maps
        pitch = Dvp * 2 + 16; ldw = kcap + 1; ldh = kcap + 8;
        v = 0;
        q = mma ? kcap * pitch : 0;
        w = q + rows * Dp * (mma ? 2 : 4);
        hi = (w + rows * ldw * 4 + 15) & ~15;
        lo = hi + (mma ? rows * ldh * 2 : 0);
        ml = lo + (mma ? rows * ldh * 2 : 0);
        krow = ml + rows * 8;
        total = krow + kcap * 4;
    }
};

__global__ void __launch_bounds__(WR_THREADS) window_rows_mma_kernel(const __grid_constant__ WindowRows P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const PtbWindowAttn& A = P.A;
    const int RB1 = (P.hg + 7) / 8, RB = RB1 * A.maps, R8 = RB1 * 8, rows = RB * 8;
    const WindowSmem L(rows, A.Dp, A.Dvp, P.kcap, true);
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem + L.q);
    float* w_s = reinterpret_cast<float*>(smem + L.w);
    __nv_bfloat16* hi_s = reinterpret_cast<__nv_bfloat16*>(smem + L.hi);
    __nv_bfloat16* lo_s = reinterpret_cast<__nv_bfloat16*>(smem + L.lo);
    float2* ml_s = reinterpret_cast<float2*>(smem + L.ml);
    int* krow = reinterpret_cast<int*>(smem + L.krow);
    const int split = blockIdx.x, i = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const HeadGroup hg = head_group(P);
    const int c = hg.c;
    pdl_wait();
    pdl_launch_dependents();
    Distance dist;
    const int nk = row_keys(P, i, split, krow, dist);
    {
        const int ch = A.Dp / 8;
        const uint4* src = reinterpret_cast<const uint4*>((const __nv_bfloat16*)A.q + ((size_t)i * A.H + hg.h0) * A.maps * A.Dp);
        uint4* dst = reinterpret_cast<uint4*>(q_s);
        for (int e = threadIdx.x; e < rows * ch; e += WR_THREADS) {
            const int row = e / ch, m = row / R8, r = row % R8;
            dst[e] = r < hg.n ? src[(r * A.maps + m) * ch + e % ch] : make_uint4(0, 0, 0, 0);
        }
    }
    __syncthreads();
    const int kgroups = (nk + 15) / 16;
    {                                                  // the values, while the scores are formed
        const int vch = A.Dvp / 8;
        const uint32_t v0 = smem_u32(smem + L.v);
        for (int e = threadIdx.x; e < kgroups * 16 * vch; e += WR_THREADS) {
            const int r = e / vch, ch = e % vch, kr = krow[r];
            fa::cp_async16(v0 + (uint32_t)(r * L.pitch + ch * 16), (const __nv_bfloat16*)A.v_pages + (kr >= 0 ? cache_row(kr, A.G, c) * A.v_ld + ch * 8 : 0), kr >= 0);
        }
        fa::cp_async_commit();
    }
    // a lane's 16 bytes serve as its elements of two k16 steps of both operands, so the order inside a 32-element group cancels
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    const int nch = A.Dp / 8, kpitch = A.maps * A.Dp;
    for (int u = warp; u < RB * kgroups; u += WR_WARPS) {
        const int kg = u % kgroups, rb = u / kgroups;
        const __nv_bfloat16* kp = (const __nv_bfloat16*)A.k_pages + (rb / RB1) * A.Dp;
        const int r0 = krow[kg * 16 + g], r1 = krow[kg * 16 + g + 8];
        const uint4* k0 = reinterpret_cast<const uint4*>(kp + cache_row(max(r0, 0), A.G, c) * kpitch);
        const uint4* k1 = reinterpret_cast<const uint4*>(kp + cache_row(max(r1, 0), A.G, c) * kpitch);
        const uint4* qv = reinterpret_cast<const uint4*>(q_s + (size_t)(rb * 8 + g) * A.Dp);
        float acc[4] = {0.f, 0.f, 0.f, 0.f};
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
                    const uint4 q4 = ch < nch ? qv[ch] : zero4;
                    const uint32_t f0[4] = {a[s].x, b[s].x, a[s].y, b[s].y}, f1[4] = {a[s].z, b[s].z, a[s].w, b[s].w};
                    fa::mma16816(acc, f0, q4.x, q4.y);
                    fa::mma16816(acc, f1, q4.z, q4.w);
                }
            }
        }
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int row = rb * 8 + 2 * t + (e & 1), j = kg * 16 + g + (e >> 1) * 8;
            float s = acc[e] * P.scale_log2;
            if (A.rel && row % R8 < hg.n) s += rel_log2(A, hg.h0 + row % R8, dist(j));
            w_s[row * L.ldw + j] = ((e >> 1) ? r1 : r0) >= 0 ? s : -INFINITY;
        }
    }
    __syncthreads();
    for (int h = warp; h < rows; h += WR_WARPS) {
        float m = -INFINITY, l = 0.f;
        for (int j = lane; j < kgroups * 16; j += 32) m = fmaxf(m, w_s[h * L.ldw + j]);
        m = warp_max(m);
        const float base = m == -INFINITY ? 0.f : m;
        for (int j = lane; j < kgroups * 16; j += 32) {
            const float p = h % R8 < hg.n ? exp2f(w_s[h * L.ldw + j] - base) : 0.f;
            const __nv_bfloat16 hi = __float2bfloat16_rn(p);
            hi_s[h * L.ldh + j] = hi;
            lo_s[h * L.ldh + j] = __float2bfloat16_rn(p - __bfloat162float(hi));
            l += p;
        }
        l = warp_sum(l);
        if (lane == 0) ml_s[h] = make_float2(m, l);
    }
    fa::cp_async_wait<0>();
    __syncthreads();
    // rows 0-7 of the left operand carry the high halves of eight heads' weights, rows 8-15 the low halves; columns are values
    const uint32_t v0 = smem_u32(smem + L.v);
    const int DC = (A.Dvp + 31) / 32;
    const bool merged = A.nsplit > 1 || A.maps > 1;
    for (int u = warp; u < RB * DC; u += WR_WARPS) {
        const int dc = u % DC, rb = u / DC;
        const bool two = dc * 32 + 16 < A.Dvp;         // Dvp is a multiple of 16
        const __nv_bfloat16* hi_r = hi_s + (rb * 8 + g) * L.ldh + 2 * t;
        const __nv_bfloat16* lo_r = lo_s + (rb * 8 + g) * L.ldh + 2 * t;
        float acc[4][4];
#pragma unroll
        for (int e = 0; e < 4; ++e)
#pragma unroll
            for (int k = 0; k < 4; ++k) acc[e][k] = 0.f;
        for (int kg = 0; kg < kgroups; ++kg) {
            uint32_t a[4];
            a[0] = *reinterpret_cast<const uint32_t*>(hi_r + kg * 16);
            a[1] = *reinterpret_cast<const uint32_t*>(lo_r + kg * 16);
            a[2] = *reinterpret_cast<const uint32_t*>(hi_r + kg * 16 + 8);
            a[3] = *reinterpret_cast<const uint32_t*>(lo_r + kg * 16 + 8);
            const uint32_t at = v0 + (uint32_t)((kg * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * L.pitch + (dc * 4 + (lane >> 4)) * 16);
            uint32_t b[4];
            fa::ldsm4_t(at, b[0], b[1], b[2], b[3]);
            fa::mma16816(acc[0], a, b[0], b[1]);
            fa::mma16816(acc[1], a, b[2], b[3]);
            if (two) {
                fa::ldsm4_t(at + 32, b[0], b[1], b[2], b[3]);
                fa::mma16816(acc[2], a, b[0], b[1]);
                fa::mma16816(acc[3], a, b[2], b[3]);
            }
        }
        const int row = rb * 8 + g, hl = row % R8, h = hg.h0 + hl;
        if (hl >= hg.n) continue;
        const float2 ml = ml_s[row];
        const float f = merged ? 1.f : finish_factor<__nv_bfloat16>(A, i, h, ml.x, ml.y);
        float* wk = A.work + ((((size_t)i * A.nsplit + split) * A.H + h) * A.maps + row / R8) * (A.Dvp + 2);
        __nv_bfloat16* o = (__nv_bfloat16*)A.out + ((size_t)i * A.H + h) * A.Dv;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int d = dc * 32 + e * 8 + 2 * t;
            const float x = acc[e][0] + acc[e][2], y = acc[e][1] + acc[e][3];
            if (merged) {
                if (d < A.Dvp) *reinterpret_cast<float2*>(wk + d) = make_float2(x, y);
            } else {
                if (d < A.Dv) o[d] = __float2bfloat16_rn(x * f);
                if (d + 1 < A.Dv) o[d + 1] = __float2bfloat16_rn(y * f);
            }
        }
        if (merged && dc == 0 && t == 0) *reinterpret_cast<float2*>(wk + A.Dvp) = ml;
    }
}

__global__ void __launch_bounds__(WR_THREADS) window_rows_f32_kernel(const __grid_constant__ WindowRows P) {
    extern __shared__ __align__(16) unsigned char smem[];
    const PtbWindowAttn& A = P.A;
    const int R8 = (P.hg + 7) / 8 * 8;
    const WindowSmem L(R8 * A.maps, A.Dp, A.Dvp, P.kcap, false);
    float* q_s = reinterpret_cast<float*>(smem + L.q);                 // [maps][n][Dp], the other arrays likewise
    float* w_s = reinterpret_cast<float*>(smem + L.w);
    float2* ml_s = reinterpret_cast<float2*>(smem + L.ml);
    int* krow = reinterpret_cast<int*>(smem + L.krow);
    const int split = blockIdx.x, i = blockIdx.z, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const HeadGroup hg = head_group(P);
    const int c = hg.c, rows = hg.n * A.maps, kpitch = A.maps * A.Dp;
    pdl_wait();
    pdl_launch_dependents();
    Distance dist;
    const int nk = row_keys(P, i, split, krow, dist);
    for (int e = threadIdx.x; e < rows * A.Dp; e += WR_THREADS) {
        const int row = e / A.Dp, m = row / hg.n, r = row % hg.n;
        q_s[e] = ((const float*)A.q)[(((size_t)i * A.H + hg.h0 + r) * A.maps + m) * A.Dp + e % A.Dp];
    }
    __syncthreads();
    for (int e = threadIdx.x; e < rows * nk; e += WR_THREADS) {
        const int h = e / nk, j = e % nk, r = krow[j];
        float s = -INFINITY;
        if (r >= 0) {
            const float4* k4 = reinterpret_cast<const float4*>((const float*)A.k_pages + cache_row(r, A.G, c) * kpitch + (h / hg.n) * A.Dp);
            const float4* q4 = reinterpret_cast<const float4*>(q_s + (size_t)h * A.Dp);
            float4 a = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int d = 0; d < A.Dp / 4; ++d) {
                const float4 x = k4[d], y = q4[d];
                a.x = fmaf(x.x, y.x, a.x); a.y = fmaf(x.y, y.y, a.y); a.z = fmaf(x.z, y.z, a.z); a.w = fmaf(x.w, y.w, a.w);
            }
            s = ((a.x + a.y) + (a.z + a.w)) * P.scale_log2;
            if (A.rel) s += rel_log2(A, hg.h0 + h % hg.n, dist(j));
        }
        w_s[h * L.ldw + j] = s;
    }
    __syncthreads();
    for (int h = warp; h < rows; h += WR_WARPS) {
        float m = -INFINITY, l = 0.f;
        for (int j = lane; j < nk; j += 32) m = fmaxf(m, w_s[h * L.ldw + j]);
        m = warp_max(m);
        for (int j = lane; j < nk; j += 32) {
            const float p = exp2f(w_s[h * L.ldw + j] - (m == -INFINITY ? 0.f : m));
            w_s[h * L.ldw + j] = p;
            l += p;
        }
        l = warp_sum(l);
        if (lane == 0) ml_s[h] = make_float2(m, l);
    }
    __syncthreads();
    const bool merged = A.nsplit > 1 || A.maps > 1;
    for (int e = threadIdx.x; e < rows * A.Dvp; e += WR_THREADS) {
        const int row = e / A.Dvp, d = e % A.Dvp, h = hg.h0 + row % hg.n;
        float a = 0.f;
        for (int j = 0; j < nk; ++j)
            if (krow[j] >= 0) a = fmaf(w_s[row * L.ldw + j], ((const float*)A.v_pages)[cache_row(krow[j], A.G, c) * A.v_ld + d], a);
        const float2 ml = ml_s[row];
        float* wk = A.work + ((((size_t)i * A.nsplit + split) * A.H + h) * A.maps + row / hg.n) * (A.Dvp + 2);
        if (merged) {
            wk[d] = a;
            if (d == 0) *reinterpret_cast<float2*>(wk + A.Dvp) = ml;
        } else if (d < A.Dv) ((float*)A.out)[((size_t)i * A.H + h) * A.Dv + d] = a * finish_factor<float>(A, i, h, ml.x, ml.y);
    }
}

// One CTA per (head, row, and with one map `cols` columns): the factor of every split first, its lanes over the splits; then `share` warps per
// map take the splits of 64 columns together, the warps left over other columns, and their sums meet in shared memory.
constexpr int WM_THREADS = 256, WM_WARPS = WM_THREADS / 32, WM_COLS = 64;
template <typename T, int MAPS>
__global__ void __launch_bounds__(WM_THREADS) window_merge_kernel(const __grid_constant__ PtbWindowAttn P, int cols, int share) {
    extern __shared__ float part_s[];                  // [MAPS share][cols] partial sums, then [MAPS][nsplit] factors
    __shared__ float red[WM_WARPS];
    const int c0 = blockIdx.z * cols, parts = MAPS * share;
    float* fac = part_s + parts * cols;
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.x, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const size_t i = blockIdx.y, pitch = (size_t)P.H * MAPS * (P.Dvp + 2);
    const float* wk = P.work + i * P.nsplit * pitch + (size_t)(h * MAPS) * (P.Dvp + 2);
    if (warp < MAPS) {                                 // a warp per map
        const float* ml = wk + (size_t)warp * (P.Dvp + 2) + P.Dvp;
        float M = -INFINITY, l = 0.f;
        for (int s = lane; s < P.nsplit; s += 32) M = fmaxf(M, ml[s * pitch]);
        M = warp_max(M);
        const float base = M == -INFINITY ? 0.f : M;
        for (int s = lane; s < P.nsplit; s += 32) {
            const float e = exp2f(ml[s * pitch] - base);
            fac[warp * P.nsplit + s] = e;
            l += ml[s * pitch + 1] * e;
        }
        l = warp_sum(l);
        const float f = MAPS == 1 ? finish_factor<T>(P, i, h, M, l) : l > 0.f ? (warp ? -P.mix : 1.f) / l : 0.f;
        __syncwarp();
        for (int s = lane; s < P.nsplit; s += 32) fac[warp * P.nsplit + s] *= f;
    }
    __syncthreads();
    const int m = warp % MAPS, mine = warp / MAPS % share;
    const float* f = fac + m * P.nsplit;
    for (int c = warp / parts * WM_COLS; c < cols; c += WM_WARPS / parts * WM_COLS) {
        const int d = c0 + c + lane * 2;               // elements d and d + 1 (Dvp is even)
        float2 r = make_float2(0.f, 0.f);
        if (d < P.Dvp) {
            const float* p = wk + (size_t)m * (P.Dvp + 2) + d;
#pragma unroll 8
            for (int s = mine; s < P.nsplit; s += share) {
                const float2 v = *reinterpret_cast<const float2*>(p + s * pitch);
                r.x = fmaf(v.x, f[s], r.x);
                r.y = fmaf(v.y, f[s], r.y);
            }
        }
        *reinterpret_cast<float2*>(part_s + warp % parts * cols + c + lane * 2) = r;
    }
    __syncthreads();
    T* out = (T*)P.out + (i * P.H + h) * P.Dv;
    float ss = 0.f;
    for (int c = threadIdx.x; c < cols; c += WM_THREADS) {
        float v = 0.f;
        for (int w = 0; w < parts; ++w) v += part_s[w * cols + c];
        if (c0 + c >= P.Dv) v = 0.f;
        if constexpr (MAPS == 1) {
            if (c0 + c < P.Dv) out[c0 + c] = wa_t<T>(v);
        } else {
            part_s[c] = v;                               // the same thread reads it again
            ss += v * v;
        }
    }
    if constexpr (MAPS == 2) {
        ss = warp_sum(ss);
        if (lane == 0) red[warp] = ss;
        __syncthreads();
        ss = 0.f;
#pragma unroll
        for (int w = 0; w < WM_WARPS; ++w) ss += red[w];
        float g = rsqrtf(ss / (float)P.Dv + P.mix_eps) * P.mix_gain;
        if (P.gate) g *= sigmoid(wa_f<T>(((const T*)P.gate)[i * P.gate_ld + h]));
        for (int c = threadIdx.x; c < P.Dv; c += WM_THREADS) out[c] = wa_t<T>(part_s[c] * g);
    }
}

}  // namespace ptb

using namespace ptb;

// After the packed projection x [n, *] (pitch ld; q, k and v rows at the three columns): q_out [n, H, Dp] = q / rms(q) * qw over all H D
// columns together; k, normed over its G D columns with kw, and v go to the page slot of (req, pos).  Dp, Dvp: sizes as stored,
// multiples of 16; the pad is zero.
PTB_API int ptb_proj_norm_write(const void* x, long long ld, int q_col, int k_col, int v_col, void* q_out, void* k_pages, void* v_pages,
                                const float* qw, const float* kw, const int* pos, int pos_stride, const int* req, int req_stride,
                                const int* page_table, int pt_stride, int n_pages, int n, int H, int G, int D, int Dp, int Dv, int Dvp, float eps,
                                int* status, int bf16, cudaStream_t st) {
    if (n <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || D <= 0 || Dv <= 0 || Dp % 16 || Dvp % 16 || Dp < D || Dvp < Dv) {
        ptb_set_error("proj_norm_write: bad sizes (H %d, G %d, D %d/%d, Dv %d/%d)", H, G, D, Dp, Dv, Dvp);
        return -1;
    }
    ProjNormParams p{x, ld, q_col, k_col, v_col, q_out, k_pages, v_pages, qw, kw, pos, req, page_table, pos_stride, req_stride, pt_stride, n_pages,
                     H, G, D, Dp, Dv, Dvp, eps, status};
    const bool vec = D % 8 == 0 && Dv % 8 == 0 && ld % 8 == 0 && q_col % 8 == 0 && k_col % 8 == 0 && v_col % 8 == 0 && ((uintptr_t)x & 15) == 0;
    const bool pdl = ptb_pdl_enabled();
    if (bf16) PTB_CUDA_OK(ptb_launch(vec ? proj_norm_write_kernel<__nv_bfloat16, 8> : proj_norm_write_kernel<__nv_bfloat16, 1>, dim3(n), dim3(PN_THREADS), 0, st, pdl, p));
    else PTB_CUDA_OK(ptb_launch(proj_norm_write_kernel<float, 1>, dim3(n), dim3(PN_THREADS), 0, st, pdl, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// Joins the splits and maps that row kernels left in a.work.
int ptb_window_merge(const PtbWindowAttn& a, cudaStream_t st) {
    auto merge = a.bf16 ? (a.maps > 1 ? window_merge_kernel<__nv_bfloat16, 2> : window_merge_kernel<__nv_bfloat16, 1>)
                        : (a.maps > 1 ? window_merge_kernel<float, 2> : window_merge_kernel<float, 1>);
    int share = 1;
    while (share * 2 * a.maps <= WM_WARPS && share * 8 <= a.nsplit) share *= 2;
    const int padded = (a.Dv + WM_COLS - 1) / WM_COLS * WM_COLS, cols = a.maps == 1 && share * a.maps == WM_WARPS ? WM_COLS : padded;
    const size_t smem = ((size_t)a.maps * share * cols + (size_t)a.maps * a.nsplit) * 4;
    if (smem > 200 * 1024) { ptb_set_error("window attention: %d splits, heads of %d", a.nsplit, a.Dv); return -1; }
    if (smem > 48 * 1024) PTB_CUDA_OK(cudaFuncSetAttribute(merge, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024));
    PTB_CUDA_OK(ptb_launch(merge, dim3(a.H, a.n, padded / cols), dim3(WM_THREADS), smem, st, ptb_pdl_enabled(), a, cols, share));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// Floats of workspace the row kernels need (heads: H times the number of maps) where nsplit or the number of maps is above one.
PTB_API long long ptb_window_rows_work_floats(int n, int heads, int Dvp, int nsplit) { return (long long)n * nsplit * heads * (Dvp + 2); }

// Query rows, each at its own position of its own sequence, against the cached keys it sees; see PtbWindowAttn.  max_keys: the most keys
// any row sees; nsplit CTAs share a row's keys (at most WA_KEYS each).
PTB_API int ptb_window_attn_rows(const PtbWindowAttn* args, cudaStream_t st) {
    const PtbWindowAttn& a = *args;
    if (a.n <= 0) return 0;
    if (a.G <= 0 || a.H % a.G || a.Dp % 16 || a.Dvp % 16 || a.v_ld % 8 || a.window < 1 || a.keep < 0 || a.maps < 1 || a.maps > 2 || (a.maps > 1 && a.sink) || (a.rel && a.rel_n < 1)) {
        ptb_set_error("window attention: bad sizes (H %d, G %d, Dp %d, Dvp %d, window %d, keep %d, maps %d)", a.H, a.G, a.Dp, a.Dvp, a.window, a.keep, a.maps);
        return -1;
    }
    const int per = (std::max(1, a.max_keys) + a.nsplit - 1) / std::max(1, a.nsplit);
    const bool merged = a.nsplit > 1 || a.maps > 1;
    if (a.nsplit < 1 || per > WA_KEYS || (merged && !a.work)) {
        ptb_set_error("window attention: %d splits for %d keys (at most %d keys per split, workspace needed above one)", a.nsplit, a.max_keys, WA_KEYS);
        return -1;
    }
    WindowRows p;
    p.A = a;
    p.kcap = (per + 15) & ~15;
    p.scale_log2 = a.scale * WA_LOG2E;
    const int R = a.H / a.G;
    p.hg = std::min(R, WA_HEADS);
    p.groups = (R + p.hg - 1) / p.hg;
    if (a.n > 65535 || a.G * p.groups > 65535) { ptb_set_error("window attention: %d rows of %d groups of heads in one launch", a.n, a.G * p.groups); return -1; }
    const WindowSmem L((p.hg + 7) / 8 * 8 * a.maps, a.Dp, a.Dvp, p.kcap, a.bf16 != 0);
    if (L.total > 227 * 1024) { ptb_set_error("window attention: %d heads of %d / %d need %d bytes of shared memory", p.hg, a.Dp, a.Dvp, L.total); return -1; }
    auto kern = a.bf16 ? window_rows_mma_kernel : window_rows_f32_kernel;
    if (L.total > 48 * 1024) PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    const bool pdl = ptb_pdl_enabled();
    PTB_CUDA_OK(ptb_launch(kern, dim3(a.nsplit, a.G * p.groups, a.n), dim3(WR_THREADS), (size_t)L.total, st, pdl, p));
    return merged ? ptb_window_merge(a, st) : 0;
}
