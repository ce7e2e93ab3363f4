// Latent attention (a cache row serves every head as key and, in its first part, as value):
//   head_linear_kernel       a matrix per head: folds W_uk into the queries (and appends their rotated part), applies W_uv to weighted
//                            latents (and the gate).  Any size, fp32 arithmetic;
//   head_linear_mma_kernel   the same on the tensor cores, bf16;
//   latent_rows_kernel       few query rows, bf16: a CTA takes up to 32 heads of a row and a share of its pages, which arrive by TMA once
//                            for both products;
//   latent_gather_kernel     the cached rows of whole contexts, laid out flat for the prompt tiles.
#include "window_attn.cuh"
#include "flash_attn.cuh"
#include "gemm_sm100.cuh"
#include <algorithm>

int ptb_make_tmap_bf16(CUtensorMap* map, const void* base, long long inner, long long outer, long long ld, int box_inner, int box_outer);
int ptb_window_merge(const PtbWindowAttn& a, cudaStream_t st);

namespace ptb {
namespace la {

struct HeadLinear {
    const void* x;                     // [n] rows of pitch ldx, head h at h * xs: K elements
    long long ldx;
    int xs;
    const void* w;                     // [H][N][K]
    int H, N, K;
    void* out;                         // [n] rows of pitch ldo, head h at h * os
    long long ldo;
    int os, n;
    const void* gate;                  // [n][H] of pitch gate_ld, or null: its sigmoid scales the head
    long long gate_ld;
    int rot_at, rot;                   // rot_at > 0: zeros from N to rot_at, then the `rot` elements behind x's K rotated, then zeros up to os
    const float* cos;
    const float* sin;
    int positions;
    const int* pos;
    int pos_stride;
    int* status;
};

constexpr int HL_THREADS = 128, HL_ROWS = 4, HL_COLS = 32;

// The columns of a head from N on for rows r0 .. r0 + rows: zeros up to rot_at, the rotated part, zeros.
template <typename T>
__device__ __forceinline__ void rotated_columns(const HeadLinear& P, int h, int r0, int rows) {
    const int pairs = P.rot / 2, zeros = P.os - P.N - P.rot;
#pragma unroll 4
    for (int e = threadIdx.x; e < rows * pairs; e += HL_THREADS) {
        const int r = r0 + e / pairs, d = e % pairs;
        int pos = P.pos[(size_t)r * P.pos_stride];
        if (pos < 0 || pos >= P.positions) {
            if (P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
            pos = 0;
        }
        const T* x = (const T*)P.x + (size_t)r * P.ldx + (size_t)h * P.xs + P.K + 2 * d;
        T* out = (T*)P.out + (size_t)r * P.ldo + (size_t)h * P.os + P.rot_at + 2 * d;
        const float c = P.cos[(size_t)pos * pairs + d], s = P.sin[(size_t)pos * pairs + d], u = (float)x[0], v = (float)x[1];
        out[0] = (T)(u * c - v * s);
        out[1] = (T)(v * c + u * s);
    }
    for (int e = threadIdx.x; e < rows * zeros; e += HL_THREADS) {
        const int r = r0 + e / zeros, k = e % zeros, c = P.N + k < P.rot_at ? P.N + k : P.N + k + P.rot;
        ((T*)P.out)[(size_t)r * P.ldo + (size_t)h * P.os + c] = (T)0.f;
    }
}

// HL_ROWS rows x HL_COLS outputs of one head per CTA: a warp takes eight outputs, its lanes share K.  The last column block pads and rotates.
template <typename T>
__global__ void __launch_bounds__(HL_THREADS) head_linear_kernel(const __grid_constant__ HeadLinear P) {
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, r0 = blockIdx.z * HL_ROWS, blocks = (P.N + HL_COLS - 1) / HL_COLS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = min(HL_ROWS, P.n - r0);
    if ((int)blockIdx.x == blocks) {
        rotated_columns<T>(P, h, r0, rows);
        return;
    }
    const int n0 = blockIdx.x * HL_COLS + warp * 8;
    float acc[HL_ROWS][8];
#pragma unroll
    for (int r = 0; r < HL_ROWS; ++r)
#pragma unroll
        for (int c = 0; c < 8; ++c) acc[r][c] = 0.f;
    const T* x = (const T*)P.x + (size_t)r0 * P.ldx + (size_t)h * P.xs;
    const T* w = (const T*)P.w + (size_t)h * P.N * P.K;
    for (int k = lane; k < P.K; k += 32) {
        float xv[HL_ROWS];
#pragma unroll
        for (int r = 0; r < HL_ROWS; ++r) xv[r] = r < rows ? (float)x[(size_t)r * P.ldx + k] : 0.f;
#pragma unroll
        for (int c = 0; c < 8; ++c)
            if (n0 + c < P.N) {
                const float f = (float)w[(size_t)(n0 + c) * P.K + k];
#pragma unroll
                for (int r = 0; r < HL_ROWS; ++r) acc[r][c] = fmaf(xv[r], f, acc[r][c]);
            }
    }
#pragma unroll
    for (int r = 0; r < HL_ROWS; ++r)
#pragma unroll
        for (int c = 0; c < 8; ++c) {
            float v = warp_sum(acc[r][c]);
            if (lane == 0 && r < rows && n0 + c < P.N) {
                if (P.gate) v *= sigmoid((float)((const T*)P.gate)[(size_t)(r0 + r) * P.gate_ld + h]);
                ((T*)P.out)[(size_t)(r0 + r) * P.ldo + (size_t)h * P.os + n0 + c] = (T)v;
            }
        }
}

constexpr int HM = 16;                 // rows and columns of a CTA of the tensor-core form

// 16 rows x 16 outputs of one head per CTA, four warps share K.  A lane's 16 bytes serve as its elements of two k16 steps of both operands,
// so the order inside a group of 32 elements cancels.
__global__ void __launch_bounds__(HL_THREADS) head_linear_mma_kernel(const __grid_constant__ HeadLinear P) {
    __shared__ float red[4][HM][HM + 1];
    const int h = blockIdx.y, r0 = blockIdx.z * HM, n0 = blockIdx.x * HM, warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int rows = min(HM, P.n - r0);
    pdl_wait();
    pdl_launch_dependents();
    if (n0 >= P.N) {
        rotated_columns<__nv_bfloat16>(P, h, r0, rows);
        return;
    }
    const __nv_bfloat16* x = (const __nv_bfloat16*)P.x + (size_t)r0 * P.ldx + (size_t)h * P.xs;
    const __nv_bfloat16* w = (const __nv_bfloat16*)P.w + ((size_t)h * P.N + n0) * P.K;
    const uint4 zero = make_uint4(0, 0, 0, 0);
    float c[2][4];
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) c[n][e] = 0.f;
#pragma unroll 4
    for (int k0 = warp * 32; k0 < P.K; k0 += 128) {
        const int k = k0 + t * 8;
        const bool in = k < P.K;
        const uint4 a0 = in && g < rows ? *reinterpret_cast<const uint4*>(x + (size_t)g * P.ldx + k) : zero;
        const uint4 a1 = in && g + 8 < rows ? *reinterpret_cast<const uint4*>(x + (size_t)(g + 8) * P.ldx + k) : zero;
        const uint32_t f0[4] = {a0.x, a1.x, a0.y, a1.y}, f1[4] = {a0.z, a1.z, a0.w, a1.w};
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            const uint4 b = in && n0 + n * 8 + g < P.N ? *reinterpret_cast<const uint4*>(w + (size_t)(n * 8 + g) * P.K + k) : zero;
            fa::mma16816(c[n], f0, b.x, b.y);
            fa::mma16816(c[n], f1, b.z, b.w);
        }
    }
#pragma unroll
    for (int n = 0; n < 2; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) red[warp][g + 8 * (e >> 1)][n * 8 + 2 * t + (e & 1)] = c[n][e];
    __syncthreads();
    for (int e = threadIdx.x; e < HM * HM; e += HL_THREADS) {
        const int r = e / HM, n = e % HM;
        if (r >= rows || n0 + n >= P.N) continue;
        float v = (red[0][r][n] + red[1][r][n]) + (red[2][r][n] + red[3][r][n]);
        if (P.gate) v *= sigmoid(__bfloat162float(((const __nv_bfloat16*)P.gate)[(size_t)(r0 + r) * P.gate_ld + h]));
        ((__nv_bfloat16*)P.out)[(size_t)(r0 + r) * P.ldo + (size_t)h * P.os + n0 + n] = __float2bfloat16_rn(v);
    }
}

// ---------------------------------------------------------------------------------------------- few query rows
constexpr int LR_THREADS = 288, PIECE = WA_PAGE * 128;       // eight warps and the producer; bytes of 64 cache rows of 64 columns

struct LatentRows {
    PtbWindowAttn A;
    int hg, groups, pieces, stages;    // heads of a CTA, CTAs per row and split, column pieces of a cache row, pages in flight
    float scale_log2;
};

// Shared memory: pages [stages][pieces][64 rows x 128 bytes], q [pieces][16 MH rows x 128 bytes] (both with the 128-byte swizzle), partial
// scores [4][16 MH][68], weights [16 MH][64] bf16, factors.
template <int MH>
struct LatentSmem {
    static constexpr int R = 16 * MH, PS = 68;
    int q, part, p, row, bar, total;
    __host__ __device__ LatentSmem(int pieces, int stages) {
        q = stages * pieces * PIECE;
        part = q + pieces * R * 128;
        p = part + 4 * R * PS * 4;
        row = p + R * 128;
        bar = row + 3 * R * 4;
        total = bar + 128 + 1024;
    }
};
__device__ __forceinline__ void rows_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }

// MH tiles of 16 heads, NB blocks of 16 value columns per warp.  Scores: warp (kq, kg) forms a quarter of the inner dimension for 32 of a
// page's keys; softmax: a row's threads add the quarters; values: a warp owns every eighth block of columns.
template <int MH, int NB>
__global__ void __launch_bounds__(LR_THREADS, 1) latent_rows_kernel(const __grid_constant__ CUtensorMap tmK, const __grid_constant__ LatentRows P) {
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    using L = LatentSmem<MH>;
    const L S(P.pieces, P.stages);
    constexpr int R = L::R, TPR = 256 / R, KPT = WA_PAGE / TPR;        // threads of a row, keys of a thread
    const PtbWindowAttn& A = P.A;
    float* part = reinterpret_cast<float*>(smem + S.part);
    float* alpha_s = reinterpret_cast<float*>(smem + S.row);
    float2* ml_s = reinterpret_cast<float2*>(alpha_s + R);
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + S.bar);
    uint64_t* empty = full + 4;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int split = blockIdx.x, h0 = blockIdx.y * P.hg, heads = min(P.hg, A.H - h0);
    const size_t i = blockIdx.z;
    if (threadIdx.x == 0) {
        for (int s = 0; s < P.stages; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 8); }
        mbar_fence_init();
        gemm::prefetch_tmap(&tmK);
    }
    pdl_wait();
    pdl_launch_dependents();
    const int pos = A.pos[i * A.pos_stride], len = max(0, pos + 1);
    if (pos < 0 && threadIdx.x == 0 && A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
    const int pages = (len + WA_PAGE - 1) / WA_PAGE, per = (pages + A.nsplit - 1) / A.nsplit, p0 = split * per, p1 = min(pages, p0 + per);
    const int* table = A.page_table + (size_t)A.req[i * A.req_stride] * A.pt_stride;
    auto page_id = [&](int p) {
        const int id = p < A.pt_stride ? table[p] : -1;
        return id >= 0 && id < A.n_pages ? id : -1;
    };
    for (int e = threadIdx.x; e < P.pieces * R * 8; e += LR_THREADS) {             // q by 16-byte chunks, zeros past the heads and the row
        const int pc = e / (R * 8), r = e / 8 % R, c = e % 8, col = pc * 64 + c * 8;
        uint4 v = make_uint4(0, 0, 0, 0);
        if (r < heads && col < A.Dp) v = *reinterpret_cast<const uint4*>((const __nv_bfloat16*)A.q + (i * A.H + h0 + r) * A.Dp + col);
        *reinterpret_cast<uint4*>(smem + S.q + pc * R * 128 + fa::tile_off<64>(r, c)) = v;
    }
    __syncthreads();
    if (warp == 8) {
        if (lane == 0) {
            bool ok = true;
            for (int p = p0, it = 0; p < p1 && ok; ++p, ++it) {
                const int s = it % P.stages, id = page_id(p);
                if (id < 0 && A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
                if (it >= P.stages) ok = mbar_wait(&empty[s], (uint32_t)((it / P.stages - 1) & 1), A.status);
                if (!ok) break;
                mbar_expect_tx(&full[s], P.pieces * PIECE);
                for (int c = 0; c < P.pieces; ++c) gemm::tma_load_2d(smem + (s * P.pieces + c) * PIECE, &tmK, c * 64, max(id, 0) * WA_PAGE, &full[s]);
            }
        }
        return;
    }
    const int kq = warp & 3, kg = warp >> 2, steps = A.Dp / 16, k_lo = steps * kq / 4, k_hi = steps * (kq + 1) / 4, blocks = A.Dvp / 16;
    const uint32_t q0 = smem_u32(smem + S.q), p_s = smem_u32(smem + S.p);
    const int row = threadIdx.x / TPR, key0 = threadIdx.x % TPR * KPT;
    float o[MH][NB][2][4];
#pragma unroll
    for (int m = 0; m < MH; ++m)
#pragma unroll
        for (int b = 0; b < NB; ++b)
#pragma unroll
            for (int e = 0; e < 8; ++e) o[m][b][e >> 2][e & 3] = 0.f;
    float m_run = -INFINITY, l_run = 0.f;
    bool ok = true;
    for (int p = p0, it = 0; p < p1; ++p, ++it) {
        const int s = it % P.stages;
        const bool there = page_id(p) >= 0;
        if (ok) ok = mbar_wait(&full[s], (uint32_t)((it / P.stages) & 1), A.status);
        const uint32_t k0 = smem_u32(smem + s * P.pieces * PIECE);
        {
            float acc[MH][4][4];
#pragma unroll
            for (int m = 0; m < MH; ++m)
#pragma unroll
                for (int e = 0; e < 16; ++e) acc[m][e >> 2][e & 3] = 0.f;
#pragma unroll 2
            for (int ks = k_lo; ks < k_hi; ++ks) {
                const uint32_t kp = k0 + (ks >> 2) * PIECE, qp = q0 + (ks >> 2) * R * 128;
                uint32_t b[2][4];
                fa::load_b<64>(kp, kg * 32, ks & 3, b[0]);
                fa::load_b<64>(kp, kg * 32 + 16, ks & 3, b[1]);
#pragma unroll
                for (int m = 0; m < MH; ++m) {
                    uint32_t a[4];
                    fa::load_a<64>(qp, m * 16, ks & 3, a);
#pragma unroll
                    for (int n = 0; n < 4; ++n) fa::mma16816(acc[m][n], a, b[n >> 1][2 * (n & 1)], b[n >> 1][2 * (n & 1) + 1]);
                }
            }
#pragma unroll
            for (int m = 0; m < MH; ++m)
#pragma unroll
                for (int n = 0; n < 4; ++n)
#pragma unroll
                    for (int e = 0; e < 2; ++e)
                        *reinterpret_cast<float2*>(part + (kq * R + m * 16 + g + 8 * e) * L::PS + kg * 32 + n * 8 + 2 * t) = make_float2(acc[m][n][2 * e], acc[m][n][2 * e + 1]);
        }
        rows_sync();
        {
            float sc[KPT], mx = -INFINITY;
#pragma unroll
            for (int j = 0; j < KPT; j += 4) {
                float4 v = *reinterpret_cast<const float4*>(part + row * L::PS + key0 + j);
#pragma unroll
                for (int k = 1; k < 4; ++k) {
                    const float4 w = *reinterpret_cast<const float4*>(part + (k * R + row) * L::PS + key0 + j);
                    v.x += w.x; v.y += w.y; v.z += w.z; v.w += w.w;
                }
                sc[j] = v.x; sc[j + 1] = v.y; sc[j + 2] = v.z; sc[j + 3] = v.w;
            }
#pragma unroll
            for (int j = 0; j < KPT; ++j) {
                sc[j] = there && p * WA_PAGE + key0 + j < len ? sc[j] * P.scale_log2 : -INFINITY;
                mx = fmaxf(mx, sc[j]);
            }
#pragma unroll
            for (int d = 1; d < TPR; d <<= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, d));
            const float m_new = fmaxf(m_run, mx), use = m_new == -INFINITY ? 0.f : m_new, alpha = exp2f(m_run - use);
            float sum = 0.f;
            uint32_t w[KPT / 2];
#pragma unroll
            for (int j = 0; j < KPT; j += 2) {
                const float a = exp2f(sc[j] - use), b = exp2f(sc[j + 1] - use);
                sum += a + b;
                w[j / 2] = fa::pack_bf16(a, b);
            }
            l_run = l_run * alpha + sum;
            m_run = m_new;
            uint8_t* dst = smem + S.p + fa::tile_off<64>(row, key0 >> 3) + (key0 & 7) * 2;
            if constexpr (KPT == 8) *reinterpret_cast<uint4*>(dst) = make_uint4(w[0], w[1], w[2], w[3]);
            else *reinterpret_cast<uint2*>(dst) = make_uint2(w[0], w[1]);
            if (key0 == 0) alpha_s[row] = alpha;
        }
        rows_sync();
        uint32_t a[MH][4][4];
#pragma unroll
        for (int m = 0; m < MH; ++m) {
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) fa::load_a<64>(p_s, m * 16, ks, a[m][ks]);
            const float f0 = alpha_s[m * 16 + g], f1 = alpha_s[m * 16 + g + 8];
#pragma unroll
            for (int b = 0; b < NB; ++b)
#pragma unroll
                for (int e = 0; e < 8; ++e) o[m][b][e >> 2][e & 3] *= (e & 2) ? f1 : f0;
        }
#pragma unroll
        for (int b = 0; b < NB; ++b) {
            const int blk = warp + 8 * b;
            if (blk < blocks) {
#pragma unroll
                for (int ks = 0; ks < 4; ++ks) {
                    uint32_t v[4];
                    fa::load_b_t<64>(k0 + (blk >> 2) * PIECE, ks * 16, (blk & 3) * 2, v);
#pragma unroll
                    for (int m = 0; m < MH; ++m) {
                        fa::mma16816(o[m][b][0], a[m][ks], v[0], v[1]);
                        fa::mma16816(o[m][b][1], a[m][ks], v[2], v[3]);
                    }
                }
            }
        }
        __syncwarp();
        if (lane == 0) mbar_arrive(&empty[s]);
    }
#pragma unroll
    for (int d = 1; d < TPR; d <<= 1) l_run += __shfl_xor_sync(0xffffffffu, l_run, d);
    if (key0 == 0) ml_s[row] = make_float2(m_run, l_run);
    rows_sync();
#pragma unroll
    for (int m = 0; m < MH; ++m)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int r = m * 16 + g + 8 * e;
            if (r >= heads) continue;
            const float2 ml = ml_s[r];
            const float f = ml.y > 0.f ? 1.f / ml.y : 0.f;
            float* wk = A.work + ((i * A.nsplit + split) * A.H + h0 + r) * (A.Dvp + 2);
            __nv_bfloat16* out = (__nv_bfloat16*)A.out + (i * A.H + h0 + r) * A.Dv;
#pragma unroll
            for (int b = 0; b < NB; ++b)
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const int c = (warp + 8 * b) * 16 + n * 8 + 2 * t;
                    if (c >= A.Dvp) continue;
                    const float x = o[m][b][n][2 * e], y = o[m][b][n][2 * e + 1];
                    if (A.nsplit > 1) *reinterpret_cast<float2*>(wk + c) = make_float2(x, y);
                    else *reinterpret_cast<uint32_t*>(out + c) = fa::pack_bf16(x * f, y * f);
                }
            if (A.nsplit > 1 && warp == 0 && t == 0) *reinterpret_cast<float2*>(wk + A.Dvp) = ml;
        }
}

template <int MH, int NB>
static int launch_rows(LatentRows p, cudaStream_t st) {
    const PtbWindowAttn& a = p.A;
    CUtensorMap mk;
    if (ptb_make_tmap_bf16(&mk, a.k_pages, a.Dp, (long long)a.n_pages * WA_PAGE, a.Dp, 64, WA_PAGE)) return -1;
    p.stages = 4;
    while (p.stages > 1 && LatentSmem<MH>(p.pieces, p.stages).total > 227 * 1024) --p.stages;
    const int smem = LatentSmem<MH>(p.pieces, p.stages).total;
    if (smem > 227 * 1024) { ptb_set_error("latent attention: a cache row of %d needs %d bytes of shared memory", a.Dp, smem); return -1; }
    PTB_CUDA_OK(cudaFuncSetAttribute(latent_rows_kernel<MH, NB>, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
    PTB_CUDA_OK(ptb_launch(latent_rows_kernel<MH, NB>, dim3(a.nsplit, p.groups, a.n), dim3(LR_THREADS), (size_t)smem, st, ptb_pdl_enabled(), mk, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
template <int MH>
static int launch_rows(const LatentRows& p, cudaStream_t st) {
    const int per_warp = (p.A.Dvp / 16 + 7) / 8;
    return per_warp <= 1 ? launch_rows<MH, 1>(p, st) : per_warp == 2 ? launch_rows<MH, 2>(p, st) : launch_rows<MH, 4>(p, st);
}

// One page of a context per CTA.
__global__ void __launch_bounds__(256) latent_gather_kernel(const uint4* __restrict__ pages, int n_pages, int vec, const int* __restrict__ table, int pt_stride, int pt_rows,
                                                            const int4* __restrict__ pieces, uint4* __restrict__ out, int rows, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    const int4 p = pieces[blockIdx.x];                 // first row, row of the page table, page of the sequence, rows
    int id = -1;
    if (p.y >= 0 && p.y < pt_rows && p.z >= 0 && p.z < pt_stride) id = table[(size_t)p.y * pt_stride + p.z];
    if (id < 0 || id >= n_pages || p.x < 0 || p.w < 0 || p.w > WA_PAGE || p.x + p.w > rows) {
        if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
        return;
    }
    const uint4* src = pages + (size_t)id * WA_PAGE * vec;
    uint4* dst = out + (size_t)p.x * vec;
#pragma unroll 4
    for (int e = threadIdx.x; e < p.w * vec; e += 256) dst[e] = src[e];
}

}  // namespace la
}  // namespace ptb

using namespace ptb;

// Query rows of latent attention, bf16; see PtbWindowAttn: k_pages holds the cache rows (G = 1, Dp elements, of which the first Dvp are the value), q
// [n, H, Dp], out [n, H, Dvp].  nsplit CTAs share a row's pages; above one, work is needed.
PTB_API int ptb_latent_attn_rows(const PtbWindowAttn* args, cudaStream_t st) {
    using namespace ptb::la;
    const PtbWindowAttn& a = *args;
    if (a.n <= 0) return 0;
    if (!a.bf16 || a.G != 1 || a.maps != 1 || a.H < 1 || a.Dp % 16 || a.Dvp % 16 || a.Dvp > 512 || a.Dvp > a.Dp || a.Dp > 640 || a.Dv != a.Dvp || a.nsplit < 1 ||
        (a.nsplit > 1 && !a.work) || a.n > 65535 || a.gate || a.sink) {
        ptb_set_error("latent attention: bad sizes (%d heads, cache row %d, value %d, %d splits, %d rows)", a.H, a.Dp, a.Dvp, a.nsplit, a.n);
        return -1;
    }
    int dev = 0;
    PTB_CUDA_OK(cudaGetDevice(&dev));
    PTB_CUDA_OK(cudaSetDevice(dev));     // the tensor-map encoder is a driver call: bind the primary context to this thread
    LatentRows p;
    p.A = a;
    p.hg = std::min(a.H, WA_HEADS);
    p.groups = (a.H + p.hg - 1) / p.hg;
    p.pieces = (a.Dp + 63) / 64;
    p.scale_log2 = a.scale * WA_LOG2E;
    if (p.hg <= 16 ? launch_rows<1>(p, st) : launch_rows<2>(p, st)) return -1;
    return a.nsplit > 1 ? ptb_window_merge(a, st) : 0;
}

// The cached rows of whole contexts: pieces [n_pieces] int4 (first row of out, row of the page table, page of the sequence, rows <= 64); out [rows,
// row], row a multiple of eight bf16 elements.
PTB_API int ptb_latent_gather(const void* pages, int n_pages, int row, const int* page_table, int pt_stride, int pt_rows, const void* pieces, int n_pieces, void* out,
                              int rows, int* status, cudaStream_t st) {
    using namespace ptb::la;
    if (n_pieces <= 0) return 0;
    if (row % 8 || (((uintptr_t)pages | (uintptr_t)out) & 15)) { ptb_set_error("latent_gather: rows of %d elements", row); return -1; }
    PTB_CUDA_OK(ptb_launch(latent_gather_kernel, dim3(n_pieces), dim3(256), 0, st, ptb_pdl_enabled(), (const uint4*)pages, n_pages, row / 8, page_table, pt_stride, pt_rows,
                           (const int4*)pieces, (uint4*)out, rows, status));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out[r, h os + n] = sum_k x[r, h xs + k] w[h, n, k] (times sigmoid(gate[r, h])) for n rows of H heads.  rot_at > 0 (a multiple of two): columns N ..
// rot_at of a head become zero, behind them come the `rot` elements of x that follow its K, rotated to the row's position, then zeros up to os.
PTB_API int ptb_head_linear(const void* x, long long ldx, int xs, const void* w, int H, int N, int K, void* out, long long ldo, int os, int n, const void* gate,
                            long long gate_ld, int rot_at, int rot, const float* cos, const float* sin, int positions, const int* pos, int pos_stride, int* status,
                            int bf16, cudaStream_t st) {
    using namespace ptb::la;
    if (n <= 0) return 0;
    if (H < 1 || H > 65535 || N < 1 || K < 1 || os < N || (rot_at > 0 && (rot_at < N || rot % 2 || rot_at + rot > os || positions < 1))) {
        ptb_set_error("head_linear: bad sizes (%d heads, %d x %d, %d at %d of %d)", H, N, K, rot, rot_at, os);
        return -1;
    }
    const bool pdl = ptb_pdl_enabled();
    for (int lo = 0; lo < n; lo += 65535 * HL_ROWS) {
        const int m = std::min(n - lo, 65535 * HL_ROWS), es = bf16 ? 2 : 4;
        HeadLinear p{(const char*)x + (size_t)lo * ldx * es, ldx, xs, w, H, N, K, (char*)out + (size_t)lo * ldo * es, ldo, os, m,
                     gate ? (const char*)gate + (size_t)lo * gate_ld * es : nullptr, gate_ld, rot_at, rot, cos, sin, positions,
                     pos ? pos + (size_t)lo * pos_stride : nullptr, pos_stride, status};
        const dim3 grid((N + HL_COLS - 1) / HL_COLS + (rot_at > 0 ? 1 : 0), H, (m + HL_ROWS - 1) / HL_ROWS);
        if (bf16 && K % 8 == 0 && xs % 8 == 0 && ldx % 8 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0)
            PTB_CUDA_OK(ptb_launch(head_linear_mma_kernel, dim3((N + HM - 1) / HM + (rot_at > 0 ? 1 : 0), H, (m + HM - 1) / HM), dim3(HL_THREADS), 0, st, pdl, p));
        else if (bf16) PTB_CUDA_OK(ptb_launch(head_linear_kernel<__nv_bfloat16>, grid, dim3(HL_THREADS), 0, st, pdl, p));
        else PTB_CUDA_OK(ptb_launch(head_linear_kernel<float>, grid, dim3(HL_THREADS), 0, st, pdl, p));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
