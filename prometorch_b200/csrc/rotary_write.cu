// After a packed projection, interleaved rotary positions and the page write (neighbours (2i, 2i + 1) turn together):
//   rope_write_kernel     rotated q, k and plain v of softmax attention;
//   latent_write_kernel   latent attention: RMS norms of the queries' and the keys' latents, the shared key part rotated;
//   latent_q_kernel       q of latent attention for the prompt tiles: own part and rotated part, each padded with zeros.
// cos / sin are fp32 tables [positions][dims / 2].  Page ids, positions and columns are checked; a bad one sets PTB_ERR_BOUNDS.
#include "window_attn.cuh"

namespace ptb {
namespace rw {

constexpr int THREADS = 256;

template <typename T> __device__ __forceinline__ float to_f(T v) { return (float)v; }
template <int E> struct Vec { float v[E]; };
template <typename T, int E>
__device__ __forceinline__ Vec<E> load(const T* p) {
    Vec<E> r;
    if constexpr (E == 8 && sizeof(T) == 2) {
        const uint4 raw = *reinterpret_cast<const uint4*>(p);
        const __nv_bfloat162* h = reinterpret_cast<const __nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) { const float2 f = __bfloat1622float2(h[e]); r.v[2 * e] = f.x; r.v[2 * e + 1] = f.y; }
    } else {
#pragma unroll
        for (int e = 0; e < E; ++e) r.v[e] = to_f<T>(p[e]);
    }
    return r;
}
template <typename T, int E>
__device__ __forceinline__ void store(T* p, const Vec<E>& r) {
    if constexpr (E == 8 && sizeof(T) == 2) {
        uint4 raw;
        __nv_bfloat162* h = reinterpret_cast<__nv_bfloat162*>(&raw);
#pragma unroll
        for (int e = 0; e < 4; ++e) h[e] = __floats2bfloat162_rn(r.v[2 * e], r.v[2 * e + 1]);
        *reinterpret_cast<uint4*>(p) = raw;
    } else {
#pragma unroll
        for (int e = 0; e < E; ++e) p[e] = (T)r.v[e];
    }
}

struct Rot {
    const float* cos;
    const float* sin;
    int dims, positions;
};
// E elements (2 or 8) of a head from element d on, d even.
template <int E>
__device__ __forceinline__ void turn(Vec<E>& f, const Rot& R, int pos, int d) {
#pragma unroll
    for (int e = 0; e < E; e += 2)
        if (d + e < R.dims) {
            const size_t at = (size_t)pos * (R.dims / 2) + (d + e) / 2;
            const float c = R.cos[at], s = R.sin[at], u = f.v[e], v = f.v[e + 1];
            f.v[e] = u * c - v * s;
            f.v[e + 1] = v * c + u * s;
        }
}

// The page-pool slot of a row's token; page -1 if it has none.  A position past the tables is an error as well.
struct Place { int pos, page, slot; };
__device__ __forceinline__ Place place_of(const int* pos_p, int pos_stride, const int* req, int req_stride, const int* table, int pt_stride, int n_pages,
                                          int positions, size_t i, int* status) {
    Place p;
    p.pos = pos_p[i * pos_stride];
    p.slot = p.pos % WA_PAGE;
    const int col = p.pos / WA_PAGE;
    p.page = -1;
    if (p.pos >= 0 && col < pt_stride && p.pos < positions) p.page = table[(size_t)req[i * req_stride] * pt_stride + col];
    if (p.page < 0 || p.page >= n_pages) {
        if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
        p.page = -1;
        p.pos = min(max(p.pos, 0), positions - 1);
    }
    return p;
}

struct RopeParams {
    const void* x;
    long long ld;
    int q_col, k_col, v_col;
    void* q_out;                       // [n][H maps][Dp], the pad filled with zeros
    void* k_pages;                     // [pages][G][64][maps Dp]
    void* v_pages;                     // [pages][G][64][Dvp]
    Rot rot;
    const int* pos;
    const int* req;
    const int* page_table;
    int pos_stride, req_stride, pt_stride, n_pages;
    int H, G, maps, D, Dp, Dv, Dvp;
    int* status;
};

// One CTA per row.  E elements per access: 8 where sizes and columns are multiples of eight, else 2 (single ones for odd sizes).
template <typename T, int E>
__global__ void __launch_bounds__(THREADS) rope_write_kernel(const __grid_constant__ RopeParams P) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = blockIdx.x;
    const Place at = place_of(P.pos, P.pos_stride, P.req, P.req_stride, P.page_table, P.pt_stride, P.n_pages, P.rot.positions, i, P.status);
    const T* row = (const T*)P.x + i * P.ld;
    // one padded head: element d of `width`, from src
    auto piece = [&](const T* src, int d, int width, bool rotated) {
        Vec<E> f;
        if (E == 8 && d < width) f = load<T, E>(src + d);
        else {
#pragma unroll
            for (int e = 0; e < E; ++e) f.v[e] = d + e < width ? to_f<T>(src[d + e]) : 0.f;
        }
        if (rotated) turn<E>(f, P.rot, at.pos, d);
        return f;
    };
    const int nq = P.H * P.maps * P.Dp;
    T* q = (T*)P.q_out + i * nq;
    for (int c = threadIdx.x * E; c < nq; c += THREADS * E) store<T, E>(q + c, piece(row + P.q_col + c / P.Dp * P.D, c % P.Dp, P.D, true));
    if (at.page < 0) return;
    const int kw = P.maps * P.Dp;
    T* k = (T*)P.k_pages + ((size_t)at.page * P.G * WA_PAGE + at.slot) * kw;
    for (int c = threadIdx.x * E; c < P.G * kw; c += THREADS * E)
        store<T, E>(k + (size_t)(c / kw) * WA_PAGE * kw + c % kw, piece(row + P.k_col + c / P.Dp * P.D, c % P.Dp, P.D, true));
    T* v = (T*)P.v_pages + ((size_t)at.page * P.G * WA_PAGE + at.slot) * P.Dvp;
    for (int c = threadIdx.x * E; c < P.G * P.Dvp; c += THREADS * E)
        store<T, E>(v + (size_t)(c / P.Dvp) * WA_PAGE * P.Dvp + c % P.Dvp, piece(row + P.v_col + c / P.Dvp * P.Dv, c % P.Dvp, P.Dv, false));
}

struct LatentParams {
    const void* x;
    long long ld;
    int dq_col, dkv_col, q_rank, rank, rot_dim;
    const float* q_w;
    const float* kv_w;
    float eps;
    Rot rot;
    void* cq;                          // [n][q_rank]
    void* pages;                       // [pages][64][row]: latent padded to rank_p, rotated part padded
    int rank_p, row;
    const int* pos;
    const int* req;
    const int* page_table;
    int pos_stride, req_stride, pt_stride, n_pages;
    int* status;
};

template <typename T, int E>
__global__ void __launch_bounds__(THREADS) latent_write_kernel(const __grid_constant__ LatentParams P) {
    __shared__ float red[2][THREADS / 32];
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = blockIdx.x;
    const Place at = place_of(P.pos, P.pos_stride, P.req, P.req_stride, P.page_table, P.pt_stride, P.n_pages, P.rot.positions, i, P.status);
    const T* q = (const T*)P.x + i * P.ld + P.dq_col;
    const T* c = (const T*)P.x + i * P.ld + P.dkv_col;
    float sq = 0.f, sc = 0.f;
    for (int e0 = threadIdx.x * E; e0 < P.q_rank; e0 += THREADS * E) {
        const Vec<E> f = load<T, E>(q + e0);
#pragma unroll
        for (int e = 0; e < E; ++e) sq += f.v[e] * f.v[e];
    }
    for (int e0 = threadIdx.x * E; e0 < P.rank; e0 += THREADS * E) {
        const Vec<E> f = load<T, E>(c + e0);
#pragma unroll
        for (int e = 0; e < E; ++e) sc += f.v[e] * f.v[e];
    }
    sq = warp_sum(sq); sc = warp_sum(sc);
    if ((threadIdx.x & 31) == 0) { red[0][threadIdx.x >> 5] = sq; red[1][threadIdx.x >> 5] = sc; }
    __syncthreads();
    sq = sc = 0.f;
#pragma unroll
    for (int w = 0; w < THREADS / 32; ++w) { sq += red[0][w]; sc += red[1][w]; }
    const float rq = rsqrtf(sq / (float)P.q_rank + P.eps), rc = rsqrtf(sc / (float)P.rank + P.eps);
    for (int e0 = threadIdx.x * E; e0 < P.q_rank; e0 += THREADS * E) {
        Vec<E> f = load<T, E>(q + e0);
#pragma unroll
        for (int e = 0; e < E; ++e) f.v[e] *= rq * P.q_w[e0 + e];
        store<T, E>((T*)P.cq + i * P.q_rank + e0, f);
    }
    if (at.page < 0) return;
    T* out = (T*)P.pages + ((size_t)at.page * WA_PAGE + at.slot) * P.row;
    for (int e0 = threadIdx.x * E; e0 < P.rank_p; e0 += THREADS * E) {
        Vec<E> f;
        if (e0 + E <= P.rank) {
            f = load<T, E>(c + e0);
#pragma unroll
            for (int e = 0; e < E; ++e) f.v[e] *= rc * P.kv_w[e0 + e];
        } else {
#pragma unroll
            for (int e = 0; e < E; ++e) f.v[e] = 0.f;
        }
        store<T, E>(out + e0, f);
    }
    for (int d = threadIdx.x * 2; d < P.row - P.rank_p; d += THREADS * 2) {        // rot_dim is even
        Vec<2> f;
        f.v[0] = d < P.rot_dim ? to_f<T>(c[P.rank + d]) : 0.f;
        f.v[1] = d < P.rot_dim ? to_f<T>(c[P.rank + d + 1]) : 0.f;
        turn<2>(f, P.rot, at.pos, d);
        store<T, 2>(out + P.rank_p + d, f);
    }
}

// q [n][H (D + rot)] of pitch ld -> out [n][H][Do + Ro]: D own elements padded to Do, the rotated rest padded to Ro.  One CTA per row.
template <typename T, int E>
__global__ void __launch_bounds__(THREADS) latent_q_kernel(const T* __restrict__ q, long long ld, T* __restrict__ out, int H, int D, int Do, int Ro, const Rot rot,
                                                           const int* __restrict__ pos_p, int pos_stride, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    const size_t i = blockIdx.x;
    int pos = pos_p[i * pos_stride];
    if (pos < 0 || pos >= rot.positions) {
        if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
        pos = 0;
    }
    const int W = Do + Ro, in = D + rot.dims;
    for (int c = threadIdx.x * E; c < H * W; c += THREADS * E) {
        const int h = c / W, d = c % W, r = d - Do;    // Do and W are multiples of 16
        const T* src = q + i * ld + h * in + (r < 0 ? d : D + r);
        const int left = r < 0 ? D - d : rot.dims - r;
        Vec<E> f;
        if (E == 8 && left >= E) f = load<T, E>(src);
        else {
#pragma unroll
            for (int e = 0; e < E; ++e) f.v[e] = e < left ? to_f<T>(src[e]) : 0.f;
        }
        if (r >= 0) turn<E>(f, rot, pos, r);
        store<T, E>(out + i * H * W + c, f);
    }
}

}  // namespace rw
}  // namespace ptb

using namespace ptb;

// x [n, *] (pitch ld): q, k and v rows at the three columns.  q_out [n, H maps, Dp]: q with the first `dims` elements of every map of every
// head rotated; k, rotated likewise, and v to the page slot of (req, pos).  Dp, Dvp: sizes as stored, multiples of 16; the pad is zero.
PTB_API int ptb_rope_write(const void* x, long long ld, int q_col, int k_col, int v_col, void* q_out, void* k_pages, void* v_pages, const float* cos,
                           const float* sin, int dims, int positions, const int* pos, int pos_stride, const int* req, int req_stride, const int* page_table,
                           int pt_stride, int n_pages, int n, int H, int G, int maps, int D, int Dp, int Dv, int Dvp, int* status, int bf16, cudaStream_t st) {
    using namespace ptb::rw;
    if (n <= 0) return 0;
    if (H <= 0 || G <= 0 || H % G || maps < 1 || D <= 0 || Dv <= 0 || Dp % 16 || Dvp % 16 || Dp < D || Dvp < Dv || dims < 0 || dims % 2 || dims > D || positions < 1) {
        ptb_set_error("rope_write: bad sizes (H %d, G %d, maps %d, D %d/%d, Dv %d/%d, %d rotated)", H, G, maps, D, Dp, Dv, Dvp, dims);
        return -1;
    }
    RopeParams p{x, ld, q_col, k_col, v_col, q_out, k_pages, v_pages, {cos, sin, dims, positions}, pos, req, page_table, pos_stride, req_stride, pt_stride, n_pages,
                 H, G, maps, D, Dp, Dv, Dvp, status};
    const bool vec = D % 8 == 0 && Dv % 8 == 0 && ld % 8 == 0 && q_col % 8 == 0 && k_col % 8 == 0 && v_col % 8 == 0 && ((uintptr_t)x & 15) == 0;
    const bool pdl = ptb_pdl_enabled();
    if (bf16) PTB_CUDA_OK(ptb_launch(vec ? rope_write_kernel<__nv_bfloat16, 8> : rope_write_kernel<__nv_bfloat16, 2>, dim3(n), dim3(THREADS), 0, st, pdl, p));
    else PTB_CUDA_OK(ptb_launch(rope_write_kernel<float, 2>, dim3(n), dim3(THREADS), 0, st, pdl, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// x [n, *] (pitch ld): the queries' latent [q_rank] at dq_col, the keys' latent [rank] and the shared key part [rot_dim] at dkv_col.  cq [n, q_rank]
// = RMS norm of the first times q_w; to the page slot of (req, pos) the row [RMS norm of the second times kv_w, rotated third], padded with
// zeros to rank_p and row.
PTB_API int ptb_latent_write(const void* x, long long ld, int dq_col, int dkv_col, int q_rank, int rank, int rot_dim, const float* q_w, const float* kv_w, float eps,
                             const float* cos, const float* sin, int positions, void* cq, void* pages, int rank_p, int row, const int* pos, int pos_stride,
                             const int* req, int req_stride, const int* page_table, int pt_stride, int n_pages, int n, int* status, int bf16, cudaStream_t st) {
    using namespace ptb::rw;
    if (n <= 0) return 0;
    if (q_rank < 1 || rank < 1 || rank_p < rank || rank_p % 16 || rot_dim < 0 || rot_dim % 2 || row - rank_p < rot_dim || row % 16 || positions < 1) {
        ptb_set_error("latent_write: bad sizes (ranks %d / %d, %d rotated, row %d)", q_rank, rank, rot_dim, row);
        return -1;
    }
    LatentParams p{x, ld, dq_col, dkv_col, q_rank, rank, rot_dim, q_w, kv_w, eps, {cos, sin, rot_dim, positions}, cq, pages, rank_p, row, pos, req, page_table,
                   pos_stride, req_stride, pt_stride, n_pages, status};
    const bool vec = q_rank % 8 == 0 && rank % 8 == 0 && ld % 8 == 0 && dq_col % 8 == 0 && dkv_col % 8 == 0 && ((uintptr_t)x & 15) == 0;
    const bool pdl = ptb_pdl_enabled();
    if (bf16) PTB_CUDA_OK(ptb_launch(vec ? latent_write_kernel<__nv_bfloat16, 8> : latent_write_kernel<__nv_bfloat16, 1>, dim3(n), dim3(THREADS), 0, st, pdl, p));
    else PTB_CUDA_OK(ptb_launch(latent_write_kernel<float, 1>, dim3(n), dim3(THREADS), 0, st, pdl, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// q [n, H (D + dims)] bf16 (pitch ld) -> out [n, H, Do + Ro]: every head's own D elements, zeros up to Do, its rotated elements, zeros up to Ro.
PTB_API int ptb_latent_q(const void* q, long long ld, void* out, int n, int H, int D, int Do, int Ro, const float* cos, const float* sin, int dims, int positions,
                         const int* pos, int pos_stride, int* status, cudaStream_t st) {
    using namespace ptb::rw;
    if (n <= 0) return 0;
    if (Do % 16 || Ro % 16 || Do < D || Ro < dims || dims % 2 || positions < 1) { ptb_set_error("latent_q: bad sizes (D %d / %d, %d rotated / %d)", D, Do, dims, Ro); return -1; }
    const bool vec = D % 8 == 0 && dims % 8 == 0 && ld % 8 == 0 && ((uintptr_t)q & 15) == 0;
    auto k = vec ? latent_q_kernel<__nv_bfloat16, 8> : latent_q_kernel<__nv_bfloat16, 2>;
    PTB_CUDA_OK(ptb_launch(k, dim3(n), dim3(THREADS), 0, st, ptb_pdl_enabled(), (const __nv_bfloat16*)q, ld, (__nv_bfloat16*)out, H, D, Do, Ro, Rot{cos, sin, dims, positions},
                           pos, pos_stride, status));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
