// Window attention (window_attn.cuh) over the many rows of a prompt, bf16, both products on the 5th-generation tensor cores.
//
// One CTA per (tile of 128 query rows of one sequence, head).  The keys a tile can see are whole pages: those of the kept first
// tokens, then those from the first row's window to the last row's position; two pages make a block of 128 keys.  Ten warps:
//   warp 8   TMA producer: the Q tile once, then the pages of K and V (the page table picks the boxes) through two-stage rings;
//   warp 9   owns tensor memory and issues the MMAs: S(j) = Q K_j^T into one of two 128-column buffers, then O_j = P_j V_j into a
//            third once the softmax warps have written P_j;
//   warps 0-7  softmax.  A thread owns one query row (its tensor-memory lane) and one of the block's two pages: scores come by
//            tcgen05.ld, the row maximum is exchanged with the partner thread through shared memory, probabilities go in bf16 to a
//            128-byte-swizzled tile (the A operand of the second product), half of the output row stays in registers.  The
//            read-back of O_{j-1} waits until the scores of block j have been reduced, so it overlaps the MMA of P_{j-1} V.
// Head sizes up to 128 (multiples of 16): the TMA fills what a 64-wide box reaches past a head with zeros.  Every wait is bounded.
// A page id outside the pool sets PTB_ERR_BOUNDS and its keys count as invisible.
#include "window_attn.cuh"
#include "gemm_sm100.cuh"

int ptb_make_tmap_bf16(CUtensorMap* map, const void* base, long long inner, long long outer, long long ld, int box_inner, int box_outer);
int ptb_make_tmap_bf16_3d(CUtensorMap* map, const void* base, long long n0, long long n1, long long n2, int b0, int b1, int b2);

namespace ptb {
namespace wa100 {

using namespace ptb::gemm;

constexpr int BQ = 128, BKV = 128, NTHREADS = 320;

struct Params {
    WindowAttnParams A;
    const int4* tiles;                 // first row, its position, rows, row of the page table
};

template <int DK, int DV>
struct Sm {
    static constexpr int Q_BYTES = BQ * DK * 2, K_BYTES = BKV * DK * 2, V_BYTES = BKV * DV * 2, P_BYTES = BQ * BKV * 2;
    static constexpr int OFF_K = Q_BYTES, OFF_V = OFF_K + 2 * K_BYTES, OFF_P = OFF_V + 2 * V_BYTES, OFF_RED = OFF_P + P_BYTES;
    static constexpr int OFF_BAR = OFF_RED + 2 * BQ * 4, TOTAL = OFF_BAR + 256 + 1024;
};

__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, int c0, int c1, int c2, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];" ::"r"(smem_u32(dst)),
                 "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
                 : "memory");
}

// The pages a tile walks, in order: `kept` leading ones, then `first`, first + 1, ...
struct Pages {
    int kept, first, count;
    __device__ __forceinline__ int at(int e) const { return e < kept ? e : first + e - kept; }
};
__device__ __forceinline__ Pages pages_of(const int4& t, int window, int keep) {
    Pages p;
    p.first = max(0, t.y - window + 1) / WA_PAGE;
    p.kept = min((keep + WA_PAGE - 1) / WA_PAGE, p.first);
    p.count = p.kept + (t.y + t.z + WA_PAGE - 1) / WA_PAGE - p.first;
    return p;
}

template <int DK, int DV>
__global__ void __launch_bounds__(NTHREADS, 1)
window_tiles_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmV,
                    const __grid_constant__ Params P) {
    using S = Sm<DK, DV>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t* sq = smem;
    uint8_t* sk = smem + S::OFF_K;
    uint8_t* sv = smem + S::OFF_V;
    uint8_t* sp = smem + S::OFF_P;
    float* red = reinterpret_cast<float*>(smem + S::OFF_RED);
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S::OFF_BAR);
    uint64_t* q_full = bars;             // [1]
    uint64_t* k_full = bars + 1;         // [2]
    uint64_t* k_empty = bars + 3;        // [2]
    uint64_t* v_full = bars + 5;         // [2]
    uint64_t* v_empty = bars + 7;        // [2]
    uint64_t* s_full = bars + 9;         // [2]
    uint64_t* p_ready = bars + 11;       // [1], 8 arrivals (one per softmax warp)
    uint64_t* o_full = bars + 12;        // [1]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 13);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);

    const WindowAttnParams& A = P.A;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, g = h / (A.H / A.G);
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < 2; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); mbar_init(&s_full[s], 1); }
        mbar_init(p_ready, 8);
        mbar_init(o_full, 1);
        *abort_flag = 0;
        mbar_fence_init();
        prefetch_tmap(&tmQ);
        prefetch_tmap(&tmK);
        prefetch_tmap(&tmV);
    }
    if (warp == 9) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    constexpr uint32_t TM_S = 0, TM_O = 256;             // column offsets: S buffers at 0 and 128, O_j at 256
    pdl_wait();
    pdl_launch_dependents();
    const int4 T = P.tiles[blockIdx.y];
    const Pages pg = pages_of(T, A.window, A.keep);
    const int nblk = (pg.count + 1) / 2;
    const int* table = A.page_table + (size_t)T.w * A.pt_stride;
    auto page_id = [&](int e) {                          // of element e of the list, or -1
        if (e >= pg.count) return -1;
        const int col = pg.at(e), id = col < A.pt_stride ? table[col] : -1;
        return id >= 0 && id < A.n_pages ? id : -1;
    };

    if (warp == 8) {
        // ---------------------------------------------------------------------------- TMA producer
        if (lane == 0 && nblk > 0) {
            bool ok = true;
            mbar_expect_tx(q_full, S::Q_BYTES);
            for (int kb = 0; kb < DK / 64; ++kb) tma_load_3d(sq + kb * (BQ * 128), &tmQ, kb * 64, h, T.x, q_full);
            for (int j = 0; j < nblk && ok; ++j) {
                const int s = j & 1;
                int row[2];
                for (int u = 0; u < 2; ++u) {
                    const int id = page_id(2 * j + u);
                    if (id < 0 && 2 * j + u < pg.count && A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
                    row[u] = (max(id, 0) * A.G + g) * WA_PAGE;
                }
                if (j >= 2) ok = mbar_wait(&k_empty[s], (uint32_t)(((j >> 1) - 1) & 1), A.status);
                if (!ok) break;
                mbar_expect_tx(&k_full[s], S::K_BYTES);
                for (int u = 0; u < 2; ++u)
                    for (int kb = 0; kb < DK / 64; ++kb)
                        tma_load_2d(sk + s * S::K_BYTES + kb * (BKV * 128) + u * 8192, &tmK, kb * 64, row[u], &k_full[s]);
                if (j >= 2) ok = mbar_wait(&v_empty[s], (uint32_t)(((j >> 1) - 1) & 1), A.status);
                if (!ok) break;
                mbar_expect_tx(&v_full[s], S::V_BYTES);
                for (int u = 0; u < 2; ++u)
                    for (int c = 0; c < DV / 64; ++c)
                        tma_load_2d(sv + s * S::V_BYTES + u * (DV / 64) * 8192 + c * 8192, &tmV, c * 64, row[u], &v_full[s]);
            }
            if (!ok) *abort_flag = 1;
        }
    } else if (warp == 9) {
        // ---------------------------------------------------------------------------- MMA issuer
        if (lane == 0 && nblk > 0) {
            constexpr uint32_t idesc_s = instr_desc(BQ, BKV, 0, 0);          // S = Q K^T: both K-major
            constexpr uint32_t idesc_o = instr_desc(BQ, DV, 0, 1);           // O = P V: P K-major, V MN-major
            bool ok = mbar_wait(q_full, 0, A.status);
            auto issue_s = [&](int j) {
                const int s = j & 1;
                if (!mbar_wait(&k_full[s], (uint32_t)((j >> 1) & 1), A.status)) return false;
                tc_fence_after();
                const uint32_t a0 = smem_u32(sq), b0 = smem_u32(sk + s * S::K_BYTES);
#pragma unroll
                for (int kb = 0; kb < DK / 64; ++kb)
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        umma_bf16(tmem_base + TM_S + (uint32_t)(s * BKV), smem_desc(a0 + kb * (BQ * 128) + k * 32, 16, 1024),
                                  smem_desc(b0 + kb * (BKV * 128) + k * 32, 16, 1024), idesc_s, (kb > 0 || k > 0) ? 1u : 0u);
                umma_commit(&k_empty[s]);
                umma_commit(&s_full[s]);
                return true;
            };
            if (ok) ok = issue_s(0);
            if (ok && nblk > 1) ok = issue_s(1);
            for (int j = 0; j < nblk && ok; ++j) {
                const int s = j & 1;
                ok = mbar_wait(p_ready, (uint32_t)(j & 1), A.status);        // P_j is in shared memory, O_{j-1} has been read
                if (ok) ok = mbar_wait(&v_full[s], (uint32_t)((j >> 1) & 1), A.status);
                if (!ok) break;
                tc_fence_after();
                const uint32_t a0 = smem_u32(sp), b0 = smem_u32(sv + s * S::V_BYTES);
#pragma unroll
                for (int hh = 0; hh < 2; ++hh)
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        umma_bf16(tmem_base + TM_O, smem_desc(a0 + hh * (BQ * 128) + k * 32, 16, 1024),
                                  smem_desc(b0 + hh * (DV / 64) * 8192 + k * 2048, 8192, 1024), idesc_o, (hh > 0 || k > 0) ? 1u : 0u);
                umma_commit(&v_empty[s]);
                umma_commit(o_full);
                if (j + 2 < nblk) ok = issue_s(j + 2);
            }
            if (!ok) *abort_flag = 1;
        }
    } else {
        // ---------------------------------------------------------------------------- softmax warps
        const int row = 32 * (warp & 3) + lane;          // query row inside the tile = tensor-memory lane
        const int hf = warp >> 2;                        // which page of a block, which DV / 2 columns of O
        const uint32_t lane_addr = tmem_base + ((uint32_t)(32 * (warp & 3)) << 16);
        const int q_pos = T.y + row, last = T.y + T.z - 1;
        float o_acc[DV / 2];
#pragma unroll
        for (int i = 0; i < DV / 2; ++i) o_acc[i] = 0.f;
        float m_run = -INFINITY, l_part = 0.f, alpha_prev = 1.f;
        bool ok = true;
        auto add_o = [&](float alpha) {                  // o_acc = o_acc * alpha + (my half of the row of O_j)
#pragma unroll
            for (int c = 0; c < DV / 64; ++c) {
                uint32_t r[32];
                tmem_ld32(lane_addr + TM_O + (uint32_t)(hf * (DV / 2) + c * 32), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) o_acc[c * 32 + i] = o_acc[c * 32 + i] * alpha + __uint_as_float(r[i]);
            }
        };
        for (int j = 0; j < nblk; ++j) {
            const int s = j & 1;
            const bool there = page_id(2 * j + hf) >= 0;
            if (ok && !*abort_flag) ok = mbar_wait(&s_full[s], (uint32_t)((j >> 1) & 1), A.status);
            else ok = false;
            tc_fence_after();
            float sc[64];
            {
                uint32_t r[32];
                tmem_ld32(lane_addr + TM_S + (uint32_t)(s * BKV + hf * 64), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) sc[i] = __uint_as_float(r[i]) * A.scale_log2;
                tmem_ld32(lane_addr + TM_S + (uint32_t)(s * BKV + hf * 64 + 32), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) sc[32 + i] = __uint_as_float(r[i]) * A.scale_log2;
            }
            const int key0 = pg.at(2 * j + hf) * WA_PAGE;
            // some row of the tile does not see all 64 keys: one lies ahead of it, or behind its window and not among the kept
            if (!there || key0 + 63 > T.y || (last - key0 >= A.window && key0 + 63 >= A.keep)) {
                const int ahead = there ? q_pos - key0 : -1, behind = q_pos - A.window - key0, kept = A.keep - key0;
#pragma unroll
                for (int i = 0; i < 64; ++i)
                    if (i > ahead || (i <= behind && i >= kept)) sc[i] = -INFINITY;
            }
            // eight independent partial maxima: a 64-long dependent chain would stall the two warps a scheduler has
            float m8[8];
#pragma unroll
            for (int i = 0; i < 8; ++i) m8[i] = sc[i];
#pragma unroll
            for (int i = 8; i < 64; ++i) m8[i & 7] = fmaxf(m8[i & 7], sc[i]);
            const float mx = fmaxf(fmaxf(fmaxf(m8[0], m8[1]), fmaxf(m8[2], m8[3])), fmaxf(fmaxf(m8[4], m8[5]), fmaxf(m8[6], m8[7])));
            red[hf * BQ + row] = mx;
            softmax_sync();
            const float m_new = fmaxf(m_run, fmaxf(red[row], red[BQ + row]));
            const float m_use = m_new == -INFINITY ? 0.f : m_new;
            const float alpha = exp2f(m_run - m_use);
            float l4[4] = {0.f, 0.f, 0.f, 0.f};
            uint32_t pk[32];
#pragma unroll
            for (int i = 0; i < 32; ++i) {
                const float p0 = exp2f(sc[2 * i] - m_use), p1 = exp2f(sc[2 * i + 1] - m_use);
                l4[i & 3] += p0 + p1;
                const __nv_bfloat162 h2 = __floats2bfloat162_rn(p0, p1);
                pk[i] = *reinterpret_cast<const uint32_t*>(&h2);
            }
            l_part = l_part * alpha + ((l4[0] + l4[1]) + (l4[2] + l4[3]));
            m_run = m_new;
            if (j > 0) {
                if (ok) ok = mbar_wait(o_full, (uint32_t)((j - 1) & 1), A.status);
                tc_fence_after();
                add_o(alpha_prev);
            }
            alpha_prev = alpha;
            // P_j -> shared memory, K-major with the 128-byte swizzle: sub-tile hf, row `row`, 16-byte chunk c at c ^ (row & 7)
            {
                uint8_t* prow = sp + hf * (BQ * 128) + row * 128;
#pragma unroll
                for (int c = 0; c < 8; ++c)
                    *reinterpret_cast<uint4*>(prow + ((c ^ (row & 7)) * 16)) = make_uint4(pk[4 * c], pk[4 * c + 1], pk[4 * c + 2], pk[4 * c + 3]);
            }
            fence_proxy_async();
            tc_fence_before();
            softmax_sync();                   // also keeps `red` from being overwritten before both partners have read it
            if (lane == 0) mbar_arrive(p_ready);
        }
        if (nblk > 0) {
            if (ok) ok = mbar_wait(o_full, (uint32_t)((nblk - 1) & 1), A.status);
            tc_fence_after();
            add_o(alpha_prev);
        }
        red[hf * BQ + row] = l_part;
        softmax_sync();
        float l = red[row] + red[BQ + row];
        if (row < T.z && T.x + row < A.n && ok) {
            float f = 1.f;
            if (A.sink) {
                const float s2 = A.sink[h] * WA_LOG2E, M = fmaxf(m_run, s2);
                f = exp2f(m_run - M);
                l = l * f + exp2f(s2 - M);
            }
            f = l > 0.f ? f / l : 0.f;
            const size_t r = (size_t)T.x + row;
            if (A.gate) f *= sigmoid(__bfloat162float(((const __nv_bfloat16*)A.gate)[r * A.gate_ld + h]));
            __nv_bfloat16* op = (__nv_bfloat16*)A.out + (r * A.H + h) * A.Dv;
            const int d0 = hf * (DV / 2);
            if ((A.Dv & 7) == 0) {
#pragma unroll
                for (int i = 0; i < DV / 2; i += 8) {
                    uint4 o;
                    __nv_bfloat162* oh = reinterpret_cast<__nv_bfloat162*>(&o);
#pragma unroll
                    for (int e = 0; e < 4; ++e) oh[e] = __floats2bfloat162_rn(o_acc[i + 2 * e] * f, o_acc[i + 2 * e + 1] * f);
                    if (d0 + i < A.Dv) *reinterpret_cast<uint4*>(op + d0 + i) = o;
                }
            } else {
#pragma unroll
                for (int i = 0; i < DV / 2; ++i)
                    if (d0 + i < A.Dv) op[d0 + i] = __float2bfloat16_rn(o_acc[i] * f);
            }
        }
        if (!ok) *abort_flag = 1;
    }
    // ---- teardown
    tc_fence_before();
    __syncthreads();
    if (warp == 9) tmem_dealloc(tmem_base, 512);
}

template <int DK, int DV>
static int launch(const Params& p, int n_tiles, cudaStream_t st) {
    const WindowAttnParams& a = p.A;
    CUtensorMap mq, mk, mv;
    if (ptb_make_tmap_bf16_3d(&mq, a.q, a.Dp, a.H, a.n, 64, 1, BQ)) return -1;
    const long long rows = (long long)a.n_pages * a.G * WA_PAGE;
    if (ptb_make_tmap_bf16(&mk, a.k_pages, a.Dp, rows, a.Dp, 64, WA_PAGE)) return -1;
    if (ptb_make_tmap_bf16(&mv, a.v_pages, a.Dvp, rows, a.Dvp, 64, WA_PAGE)) return -1;
    static bool attr = false;
    if (!attr) {
        PTB_CUDA_OK(cudaFuncSetAttribute(window_tiles_kernel<DK, DV>, cudaFuncAttributeMaxDynamicSharedMemorySize, Sm<DK, DV>::TOTAL));
        attr = true;
    }
    PTB_CUDA_OK(ptb_launch(window_tiles_kernel<DK, DV>, dim3(a.H, n_tiles), dim3(NTHREADS), (size_t)Sm<DK, DV>::TOTAL, st, ptb_pdl_enabled(), mq, mk, mv, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

}  // namespace wa100
}  // namespace ptb

// Query tiles [n_tiles] int4 (first row, its position, rows <= 128, page-table row) of q [n, H, Dp] bf16 against the pages; sizes as stored
// up to 128.  out [n, H Dv] bf16.  gate: bf16 with row pitch gate_ld, or null.
PTB_API int ptb_window_attn_tiles(const void* q, void* out, int n, const void* tiles, int n_tiles, int H, int G, int Dp, int Dv, int Dvp,
                                  const int* page_table, int pt_stride, int n_pages, const void* k_pages, const void* v_pages, const float* sink,
                                  const void* gate, long long gate_ld, int window, int keep, float scale, int* status, cudaStream_t st) {
    using namespace ptb;
    if (n <= 0 || n_tiles <= 0) return 0;
    if (G <= 0 || H % G || Dp % 16 || Dvp % 16 || Dp > 128 || Dvp > 128 || Dv > Dvp || window < 1 || keep < 0 || n_tiles > 65535 ||
        (long long)n_pages * G * WA_PAGE > 0x7fffffffLL) {
        ptb_set_error("window attention (tcgen05): bad sizes (H %d, G %d, Dp %d, Dvp %d, window %d, keep %d, %d tiles)", H, G, Dp, Dvp, window, keep, n_tiles);
        return -1;
    }
    int dev = 0;
    PTB_CUDA_OK(cudaGetDevice(&dev));
    PTB_CUDA_OK(cudaSetDevice(dev));     // the tensor-map encoder is a driver call: bind the primary context to this thread
    wa100::Params p;
    WindowAttnParams& a = p.A;
    memset(&p, 0, sizeof(p));
    a.q = q; a.out = out; a.page_table = page_table; a.k_pages = k_pages; a.v_pages = v_pages; a.sink = sink; a.gate = gate; a.gate_ld = gate_ld;
    a.pt_stride = pt_stride; a.n_pages = n_pages; a.n = n; a.H = H; a.G = G; a.Dp = Dp; a.Dv = Dv; a.Dvp = Dvp; a.window = window; a.keep = keep;
    a.scale_log2 = scale * WA_LOG2E; a.status = status;
    p.tiles = (const int4*)tiles;
    if (Dp <= 64) return Dvp <= 64 ? wa100::launch<64, 64>(p, n_tiles, st) : wa100::launch<64, 128>(p, n_tiles, st);
    return Dvp <= 64 ? wa100::launch<128, 64>(p, n_tiles, st) : wa100::launch<128, 128>(p, n_tiles, st);
}
