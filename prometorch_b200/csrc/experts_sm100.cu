// Grouped products of a mixture of experts on the 5th-generation tensor cores, bf16.  Rows are sorted by expert; the row counts are read
// from device memory, so nothing waits for the host.
//   expert_gather_kernel   the rows of the tokens in the order by expert;
//   expert_gemm_kernel     persistent CTAs walk the tiles of all experts.  320 threads: warp 0 TMA producer, warp 1 owns tensor memory and
//                          issues the MMAs, warps 2-9 epilogue; two accumulators, so an epilogue overlaps the next tile's main loop.
//     many rows per expert: 128 rows x 256 weight rows; gated, these are 128 gate rows and the 128 up rows that go with them;
//     few: the weight is the 128-row operand (gated: one tile of gate and one of up rows, two accumulators), 32 tokens are the columns.
//   Gated products leave silu(gate) * up.
// A TMA box may reach past an expert into the next one's rows; what it brings is never stored.
#include "gemm_sm100.cuh"
#include <algorithm>

int ptb_make_tmap_bf16(CUtensorMap* map, const void* base, long long inner, long long outer, long long ld, int box_inner, int box_outer);

namespace ptb {
namespace moe100 {

using namespace ptb::gemm;

constexpr int MAX_EXPERTS = 1024, WT = 128;            // WT: weight rows of a box

__global__ void __launch_bounds__(256) expert_gather_kernel(const uint4* __restrict__ h, long long ld, const int* __restrict__ token, const int* __restrict__ count,
                                                            uint4* __restrict__ out, int rows, int vec, int tokens, int* status) {
    pdl_wait();
    pdl_launch_dependents();
    rows = min(rows, *count);
    for (int r = blockIdx.x; r < rows; r += gridDim.x) {
        int t = token[r];
        if (t < 0 || t >= tokens) {
            if (threadIdx.x == 0 && status) atomicExch(status, PTB_ERR_BOUNDS);
            t = 0;
        }
        for (int c = threadIdx.x; c < vec; c += blockDim.x) out[(size_t)r * vec + c] = h[(size_t)t * ld + c];
    }
}

struct Params {
    const int* offsets;                // [E + 1]
    __nv_bfloat16* out;                // [rows][N]
    int rows, E, N, K;                 // N: outputs per row
    int* status;
};

template <bool GATED, bool SWAP>
struct Cfg {
    static constexpr int ROWS = SWAP ? 32 : 128;       // sorted rows of a tile
    static constexpr int WB = SWAP && !GATED ? 1 : 2;  // weight boxes of a k-block
    static constexpr int COLS = SWAP || GATED ? WT : 2 * WT;       // outputs per row of a tile
    static constexpr int W_BYTES = WB * WT * 128, T_BYTES = ROWS * 128, STAGE = W_BYTES + T_BYTES;
    static constexpr int STAGES = SWAP ? (GATED ? 6 : 11) : 4;
    static constexpr int ACC = SWAP ? WB * ROWS : 256; // columns of an accumulator
    static constexpr int TMEM = SWAP ? 128 : 512;
    static constexpr int BAR = STAGES * STAGE, TOTAL = BAR + 512 + (MAX_EXPERTS + 1) * 4 + 1024;
    static_assert(2 * ACC <= TMEM && TOTAL <= 227 * 1024, "sizes");
};

struct Tile { int e, row, end, col; };

template <bool GATED, bool SWAP>
__global__ void __launch_bounds__(THREADS, 1) expert_gemm_kernel(const __grid_constant__ CUtensorMap tmT, const __grid_constant__ CUtensorMap tmW,
                                                                 const __grid_constant__ Params P) {
    using C = Cfg<GATED, SWAP>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + C::BAR);
    uint64_t* empty = full + C::STAGES;
    uint64_t* acc_full = empty + C::STAGES;            // [2]
    uint64_t* acc_empty = acc_full + 2;                // [2]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(acc_empty + 2);
    int* cum = reinterpret_cast<int*>(smem + C::BAR + 512);        // tiles of the experts before
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int kblocks = (P.K + BK - 1) / BK, col_tiles = (P.N + C::COLS - 1) / C::COLS;
    if (threadIdx.x == 0) {
        for (int s = 0; s < C::STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        for (int b = 0; b < 2; ++b) { mbar_init(&acc_full[b], 1); mbar_init(&acc_empty[b], EPI_WARPS); }
        mbar_fence_init();
        prefetch_tmap(&tmT);
        prefetch_tmap(&tmW);
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, C::TMEM);
        tmem_relinquish();
    }
    pdl_wait();
    pdl_launch_dependents();
    if (warp == 0) {
        int run = 0;
        for (int e0 = 0; e0 < P.E; e0 += 32) {
            const int e = e0 + lane;
            int v = 0;
            if (e < P.E) v = (max(0, P.offsets[e + 1] - P.offsets[e]) + C::ROWS - 1) / C::ROWS * col_tiles;
            int s = v;
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const int t = __shfl_up_sync(0xffffffffu, s, o);
                if (lane >= o) s += t;
            }
            if (e < P.E) cum[e] = run + s - v;
            run += __shfl_sync(0xffffffffu, s, 31);
        }
        if (lane == 0) cum[P.E] = run;
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    const int tiles = cum[P.E];
    auto tile_of = [&](int t) {
        int lo = 0, hi = P.E;                          // the last expert whose tiles start at or before t
        while (hi - lo > 1) {
            const int mid = (lo + hi) >> 1;
            if (cum[mid] <= t) lo = mid; else hi = mid;
        }
        Tile r;
        r.e = lo;
        const int first = P.offsets[lo], left = t - cum[lo];
        r.end = min(P.offsets[lo + 1], P.rows);
        const int row_tiles = (cum[lo + 1] - cum[lo]) / col_tiles;
        r.row = first + left % row_tiles * C::ROWS;    // the tiles of one weight block follow one another
        r.col = left / row_tiles * C::COLS;
        return r;
    };
    if (warp == 0) {
        if (lane == 0) {
            bool ok = true;
            int it = 0;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x) {
                const Tile T = tile_of(t);
                const int w0 = T.e * (GATED ? 2 : 1) * P.N + T.col, w1 = w0 + (GATED ? P.N : WT);
                for (int kb = 0; kb < kblocks && ok; ++kb, ++it) {
                    const int s = it % C::STAGES;
                    if (it >= C::STAGES) ok = mbar_wait(&empty[s], (uint32_t)(((it / C::STAGES) - 1) & 1), P.status);
                    if (!ok) break;
                    uint8_t* st = smem + s * C::STAGE;
                    mbar_expect_tx(&full[s], C::STAGE);
                    tma_load_2d(st, &tmW, kb * BK, w0, &full[s]);
                    if constexpr (C::WB == 2) tma_load_2d(st + WT * 128, &tmW, kb * BK, w1, &full[s]);
                    tma_load_2d(st + C::W_BYTES, &tmT, kb * BK, T.row, &full[s]);
                }
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = SWAP ? instr_desc(WT, C::ROWS, 0, 0) : instr_desc(C::ROWS, 2 * WT, 0, 0);
            bool ok = true;
            int it = 0, tl = 0;
            for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++tl) {
                const int b = tl & 1;
                if (tl >= 2) ok = mbar_wait(&acc_empty[b], (uint32_t)(((tl >> 1) - 1) & 1), P.status);
                if (!ok) break;
                tc_fence_after();
                const uint32_t d = tmem_base + (uint32_t)(b * C::ACC);
                for (int kb = 0; kb < kblocks && ok; ++kb, ++it) {
                    const int s = it % C::STAGES;
                    ok = mbar_wait(&full[s], (uint32_t)((it / C::STAGES) & 1), P.status);
                    if (!ok) break;
                    tc_fence_after();
                    const uint32_t w = smem_u32(smem + s * C::STAGE), x = w + C::W_BYTES;
#pragma unroll
                    for (int k = 0; k < BK / UMMA_K; ++k) {
                        const uint64_t dx = smem_desc(x + k * 32, 16, 1024);
                        const uint32_t more = (kb > 0 || k > 0) ? 1u : 0u;
                        if constexpr (SWAP) {
#pragma unroll
                            for (int m = 0; m < C::WB; ++m) umma_bf16(d + m * C::ROWS, smem_desc(w + m * WT * 128 + k * 32, 16, 1024), dx, idesc, more);
                        } else umma_bf16(d, dx, smem_desc(w + k * 32, 16, 1024), idesc, more);
                    }
                    umma_commit(&empty[s]);
                }
                if (ok) umma_commit(&acc_full[b]);
            }
        }
    } else {
        const int q = warp & 3, half = warp >= 6;      // tensor-memory lanes of this warp; the half of a tile it stores
        const bool wide = P.N % 16 == 0 && ((uintptr_t)P.out & 31) == 0;
        bool ok = true;
        int tl = 0;
        for (int t = blockIdx.x; t < tiles && ok; t += gridDim.x, ++tl) {
            const Tile T = tile_of(t);
            const int b = tl & 1;
            ok = mbar_wait(&acc_full[b], (uint32_t)((tl >> 1) & 1), P.status);
            if (!ok) break;
            tc_fence_after();
            const uint32_t acc = tmem_base + ((uint32_t)(q * 32) << 16) + (uint32_t)(b * C::ACC);
            if constexpr (SWAP) {
                const int f = T.col + q * 32 + lane, n = min(C::ROWS, T.end - T.row);
                uint32_t g[32], u[32];
                tmem_ld32(acc, g);
                if constexpr (GATED) tmem_ld32(acc + C::ROWS, u);
                tmem_ld_wait();
                if (f < P.N) {                         // four warps take the even tokens, four the odd ones
                    __nv_bfloat16* o = P.out + (size_t)T.row * P.N + f;
#pragma unroll
                    for (int j = 0; j < 32; ++j)
                        if (j < n && (j & 1) == half) {
                            float v = __uint_as_float(g[j]);
                            if constexpr (GATED) v = silu(v) * __uint_as_float(u[j]);
                            o[(size_t)j * P.N] = __float2bfloat16_rn(v);
                        }
                }
            } else {
                const int row = T.row + q * 32 + lane;
                __nv_bfloat16* o = P.out + (size_t)row * P.N;
#pragma unroll 1
                for (int c = half * (C::COLS / 2); c < (half + 1) * (C::COLS / 2); c += 32) {
                    if (T.col + c >= P.N) break;
                    uint32_t g[32], u[32];
                    tmem_ld32(acc + c, g);
                    if constexpr (GATED) tmem_ld32(acc + WT + c, u);
                    tmem_ld_wait();
                    if (row < T.end) {
#pragma unroll
                        for (int j = 0; j < 32; j += 16) {     // N is a multiple of eight
                            uint4 v[2];
                            __nv_bfloat162* vh = reinterpret_cast<__nv_bfloat162*>(v);
#pragma unroll
                            for (int i = 0; i < 8; ++i) {
                                float x = __uint_as_float(g[j + 2 * i]), y = __uint_as_float(g[j + 2 * i + 1]);
                                if constexpr (GATED) { x = silu(x) * __uint_as_float(u[j + 2 * i]); y = silu(y) * __uint_as_float(u[j + 2 * i + 1]); }
                                vh[i] = __floats2bfloat162_rn(x, y);
                            }
                            __nv_bfloat16* dst = o + T.col + c + j;
                            const int left = P.N - (T.col + c + j);
                            if (left >= 16 && wide) st_global_32(dst, v[0], v[1]);
                            else {
                                if (left > 0) *reinterpret_cast<uint4*>(dst) = v[0];
                                if (left > 8) *reinterpret_cast<uint4*>(dst + 8) = v[1];
                            }
                        }
                    }
                }
            }
            tc_fence_before();
            __syncwarp();
            if (lane == 0) mbar_arrive(&acc_empty[b]);
        }
    }
    // ---- teardown: every role has left its loop (waits are bounded)
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem_base, C::TMEM);
}

template <bool GATED, bool SWAP>
static int launch(const void* a, long long lda, const void* w, const Params& p, int n_sm, cudaStream_t st) {
    using C = Cfg<GATED, SWAP>;
    CUtensorMap mt, mw;
    if (ptb_make_tmap_bf16(&mt, a, p.K, p.rows, lda, BK, C::ROWS)) return -1;
    if (ptb_make_tmap_bf16(&mw, w, p.K, (long long)p.E * (GATED ? 2 : 1) * p.N, p.K, BK, WT)) return -1;
    static bool attr = false;
    if (!attr) {
        PTB_CUDA_OK(cudaFuncSetAttribute(expert_gemm_kernel<GATED, SWAP>, cudaFuncAttributeMaxDynamicSharedMemorySize, C::TOTAL));
        attr = true;
    }
    const long long row_tiles = std::min<long long>(p.rows, p.rows / C::ROWS + p.E);
    const int grid = (int)std::min<long long>(n_sm, row_tiles * ((p.N + C::COLS - 1) / C::COLS));
    PTB_CUDA_OK(ptb_launch(expert_gemm_kernel<GATED, SWAP>, dim3(grid), dim3(THREADS), (size_t)C::TOTAL, st, ptb_pdl_enabled(), mt, mw, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

}  // namespace moe100
}  // namespace ptb

using namespace ptb;

// out [rows, W] = h[token[r]] (rows of h [tokens] of pitch ld), bf16, for the first `count` (on the device) of at most `rows` rows; W, ld multiples
// of eight, 16-byte aligned.
PTB_API int ptb_expert_gather(const void* h, long long ld, const int* token, const int* count, void* out, int rows, int W, int tokens, int* status, cudaStream_t st) {
    if (rows <= 0) return 0;
    if (W % 8 || ld % 8 || (((uintptr_t)h | (uintptr_t)out) & 15)) { ptb_set_error("expert_gather: %d columns of pitch %lld", W, ld); return -1; }
    const int vec = W / 8, threads = std::min(256, (vec + 31) / 32 * 32);
    PTB_CUDA_OK(ptb_launch(moe100::expert_gather_kernel, dim3(std::min(rows, 148 * 16)), dim3(threads), 0, st, ptb_pdl_enabled(), (const uint4*)h, ld / 8, token, count, (uint4*)out,
                           rows, vec, tokens, status));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

// out [rows, N] = A_e B_e^T for the sorted rows a [rows, K] (pitch lda) of every expert e (offsets [E + 1] on the device), bf16; `gated`: B_e has 2 N
// rows, gate rows first, and the result is silu(gate) * up.  N, K, lda multiples of eight.  few: the shape for few rows per expert.
PTB_API int ptb_expert_gemm(const void* a, long long lda, const void* b, int gated, void* out, const int* offsets, int rows, int E, int N, int K, int few, int n_sm,
                            int* status, cudaStream_t st) {
    using namespace ptb::moe100;
    if (rows <= 0 || N <= 0 || K <= 0) return 0;
    if (E < 1 || E > MAX_EXPERTS || N % 8 || K % 8 || lda % 8 || ((uintptr_t)out & 15) || (long long)E * 2 * N > 0x7fffffffLL) {
        ptb_set_error("expert_gemm: bad sizes (%d experts, %d x %d)", E, N, K);
        return -1;
    }
    int dev = 0;
    PTB_CUDA_OK(cudaGetDevice(&dev));
    PTB_CUDA_OK(cudaSetDevice(dev));     // the tensor-map encoder is a driver call: bind the primary context to this thread
    if (n_sm <= 0) PTB_CUDA_OK(cudaDeviceGetAttribute(&n_sm, cudaDevAttrMultiProcessorCount, dev));
    const moe100::Params p{offsets, (__nv_bfloat16*)out, rows, E, N, K, status};
    if (gated) return few ? launch<true, true>(a, lda, b, p, n_sm, st) : launch<true, false>(a, lda, b, p, n_sm, st);
    return few ? launch<false, true>(a, lda, b, p, n_sm, st) : launch<false, false>(a, lda, b, p, n_sm, st);
}
