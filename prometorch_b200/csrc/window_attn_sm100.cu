// Attention of window_attn.cuh over the many rows of a prompt, bf16, both products on the 5th-generation tensor cores.
//
// One CTA per (tile of 128 query rows of one sequence, head).  The keys a tile can see are whole pages: those of the kept first
// tokens, then those from the first row's lowest key to the last row's position; two pages make a block of 128 keys.  Ten warps:
//   warp 8   TMA producer: the Q tile once, then K in pieces of 64 columns through a ring, and V through two stages;
//   warp 9   owns tensor memory and issues the MMAs: S(j) = Q K_j^T into one of two 128-column buffers, then O_j = P_j V_j into a
//            third once the softmax warps have written P_j;
//   warps 0-7  softmax.  A thread owns one query row (its tensor-memory lane) and one of the block's two pages: scores come by
//            tcgen05.ld, the row maximum is exchanged with the partner thread through shared memory, probabilities go in bf16 to a
//            128-byte-swizzled tile (the A operand of the second product), half of the output row stays in registers.  The
//            read-back of O_{j-1} waits until the scores of block j have been reduced, so it overlaps the MMA of P_{j-1} V.
// Two maps are two rounds over the same blocks in one sequence of blocks; the first one's output waits in tensor memory (tcgen05.st) for
// the second's.  Keys and values come from the pages, or lie flat by context position with a column piece that all heads share (latent
// attention after its up-projections).  Sizes are multiples of 16; the TMA fills what a 64-wide box reaches past an extent with zeros.
// Every wait is bounded.  A page id outside the pool sets PTB_ERR_BOUNDS and its keys count as invisible.
#include "window_attn.cuh"
#include "gemm_sm100.cuh"

int ptb_make_tmap_bf16_3d(CUtensorMap* map, const void* base, long long n0, long long n1, long long n2, int b0, int b1, int b2);
int ptb_make_tmap_bf16_4d(CUtensorMap* map, const void* base, const long long* n, const long long* strides, const int* box);

namespace ptb {
namespace wa100 {

using namespace ptb::gemm;

constexpr int MAX_REL = 8192;          // entries of a head's distance bias (one map, keys from pages)
constexpr int BQ = 128, BKV = 128, NTHREADS = 320, SUB = BKV * 128;      // SUB: bytes of 128 rows of 64 columns

struct Params {
    PtbWindowAttn A;
    int k_own;                         // column pieces of a head's own keys; the rest is the shared part
    float scale_log2;
};

// KT pieces of 64 columns make a key; MAPS query tiles stay resident.
template <int KT, int DV, int MAPS>
struct Sm {
    static constexpr int NK = KT == 3 ? 5 : 4, V_BYTES = BKV * DV * 2, P_BYTES = BQ * BKV * 2;
    static constexpr int OFF_K = MAPS * KT * SUB, OFF_V = OFF_K + NK * SUB, OFF_P = OFF_V + 2 * V_BYTES, OFF_RED = OFF_P + P_BYTES;
    static constexpr int OFF_BAR = OFF_RED + 2 * BQ * 4, OFF_REL = OFF_BAR + 256, TOTAL = OFF_REL + 1024;        // and the head's distance bias
    static constexpr int MOST = TOTAL + (MAPS == 1 && KT < 3 ? MAX_REL * 4 : 0);
    static_assert(MOST <= 227 * 1024, "shared memory of a CTA");
};

__device__ __forceinline__ void softmax_sync() { asm volatile("bar.sync 1, 256;" ::: "memory"); }
__device__ __forceinline__ void tma_load_4d(void* dst, const CUtensorMap* map, int c0, int c1, int c2, int c3, uint64_t* bar) {
    asm volatile("cp.async.bulk.tensor.4d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5, %6}], [%2];" ::"r"(smem_u32(dst)),
                 "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2), "r"(c3)
                 : "memory");
}
__device__ __forceinline__ void tmem_st32(uint32_t taddr, const uint32_t* r) {
    asm volatile(
        "tcgen05.st.sync.aligned.32x32b.x32.b32 [%0], "
        "{%1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15, %16, "
        "%17, %18, %19, %20, %21, %22, %23, %24, %25, %26, %27, %28, %29, %30, %31, %32};" ::"r"(taddr),
        "r"(r[0]), "r"(r[1]), "r"(r[2]), "r"(r[3]), "r"(r[4]), "r"(r[5]), "r"(r[6]), "r"(r[7]), "r"(r[8]), "r"(r[9]), "r"(r[10]), "r"(r[11]),
        "r"(r[12]), "r"(r[13]), "r"(r[14]), "r"(r[15]), "r"(r[16]), "r"(r[17]), "r"(r[18]), "r"(r[19]), "r"(r[20]), "r"(r[21]), "r"(r[22]),
        "r"(r[23]), "r"(r[24]), "r"(r[25]), "r"(r[26]), "r"(r[27]), "r"(r[28]), "r"(r[29]), "r"(r[30]), "r"(r[31])
        : "memory");
}
__device__ __forceinline__ void tmem_st_wait() { asm volatile("tcgen05.wait::st.sync.aligned;" ::: "memory"); }
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
__device__ __forceinline__ Pages pages_of(const int4& t, int window, int keep, int chunked) {
    Pages p;
    p.first = low_of(t.y, window, chunked) / WA_PAGE;
    p.kept = min((keep + WA_PAGE - 1) / WA_PAGE, p.first);
    p.count = p.kept + (t.y + t.z + WA_PAGE - 1) / WA_PAGE - p.first;
    return p;
}

template <int KT, int DV, int MAPS>
__global__ void __launch_bounds__(NTHREADS, 1)
window_tiles_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ CUtensorMap tmR,
                    const __grid_constant__ CUtensorMap tmV, const __grid_constant__ Params P) {
    using S = Sm<KT, DV, MAPS>;
    constexpr int NK = S::NK;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint8_t* sq = smem;
    uint8_t* sk = smem + S::OFF_K;
    uint8_t* sv = smem + S::OFF_V;
    uint8_t* sp = smem + S::OFF_P;
    float* red = reinterpret_cast<float*>(smem + S::OFF_RED);
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + S::OFF_BAR);
    uint64_t* q_full = bars;             // [1]
    uint64_t* k_full = bars + 1;         // [NK <= 5]
    uint64_t* k_empty = bars + 6;        // [NK]
    uint64_t* v_full = bars + 11;        // [2]
    uint64_t* v_empty = bars + 13;       // [2]
    uint64_t* s_full = bars + 15;        // [2]
    uint64_t* p_ready = bars + 17;       // [1], 8 arrivals (one per softmax warp)
    uint64_t* o_full = bars + 18;        // [1]
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(bars + 19);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    float* rel = reinterpret_cast<float*>(smem + S::OFF_REL);

    const PtbWindowAttn& A = P.A;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int h = blockIdx.x, g = h / (A.H / A.G);
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int s = 0; s < NK; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
        for (int s = 0; s < 2; ++s) { mbar_init(&v_full[s], 1); mbar_init(&v_empty[s], 1); mbar_init(&s_full[s], 1); }
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
    if (A.rel)                                           // a weight of the model: no kernel before this one writes it
        for (int e = threadIdx.x; e < A.rel_n; e += NTHREADS) rel[e] = A.rel[(size_t)h * A.rel_n + e] * WA_LOG2E;
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem_base = *tmem_slot;
    constexpr uint32_t TM_S = 0, TM_O = 256, TM_KEEP = 384;      // column offsets: S buffers at 0 and 128, O_j, the first map's output
    pdl_wait();
    pdl_launch_dependents();
    const int4 T = reinterpret_cast<const int4*>(A.tiles)[blockIdx.y];
    const Pages pg = pages_of(T, A.window, A.keep, A.chunked);
    const int nblk = (pg.count + 1) / 2, total = MAPS * nblk;    // block j: keys of block j % nblk, map j / nblk
    const bool flat = A.flat_rows > 0;
    const int* table = A.page_table + (flat ? 0 : (size_t)T.w * A.pt_stride);
    auto page_id = [&](int e) {                          // of element e of the list, or -1; flat: its place in the context
        if (e >= pg.count) return -1;
        const int col = pg.at(e);
        if (flat) return col;
        const int id = col < A.pt_stride ? table[col] : -1;
        return id >= 0 && id < A.n_pages ? id : -1;
    };

    if (warp == 8) {
        // ---------------------------------------------------------------------------- TMA producer
        if (lane == 0 && nblk > 0) {
            bool ok = true;
            mbar_expect_tx(q_full, MAPS * KT * SUB);
            for (int m = 0; m < MAPS; ++m)
                for (int kb = 0; kb < KT; ++kb) tma_load_3d(sq + (m * KT + kb) * SUB, &tmQ, kb * 64, h * MAPS + m, T.x, q_full);
            int it = 0;
            for (int j = 0; j < total && ok; ++j) {
                const int s = j & 1, blk = MAPS == 1 ? j : j % nblk, m = MAPS == 1 ? 0 : j / nblk;
                int row[2], page[2];
                for (int u = 0; u < 2; ++u) {
                    const int id = page_id(2 * blk + u);
                    if (id < 0 && 2 * blk + u < pg.count && A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
                    row[u] = flat ? T.w + max(id, 0) * WA_PAGE : 0;
                    page[u] = flat ? 0 : max(id, 0);
                }
                for (int kb = 0; kb < KT && ok; ++kb, ++it) {
                    const int slot = it % NK;
                    if (it >= NK) ok = mbar_wait(&k_empty[slot], (uint32_t)(((it / NK) - 1) & 1), A.status);
                    if (!ok) break;
                    mbar_expect_tx(&k_full[slot], SUB);
                    for (int u = 0; u < 2; ++u) {
                        uint8_t* dst = sk + slot * SUB + u * 8192;
                        if (kb < P.k_own) tma_load_4d(dst, &tmK, m * A.Dp + kb * 64, row[u], g, page[u], &k_full[slot]);
                        else tma_load_4d(dst, &tmR, (kb - P.k_own) * 64, row[u], 0, 0, &k_full[slot]);
                    }
                }
                if (ok && j >= 2) ok = mbar_wait(&v_empty[s], (uint32_t)(((j >> 1) - 1) & 1), A.status);
                if (!ok) break;
                mbar_expect_tx(&v_full[s], S::V_BYTES);
                for (int u = 0; u < 2; ++u)
                    for (int c = 0; c < DV / 64; ++c)
                        tma_load_4d(sv + s * S::V_BYTES + u * (DV / 64) * 8192 + c * 8192, &tmV, c * 64, row[u], g, page[u], &v_full[s]);
            }
            if (!ok) *abort_flag = 1;
        }
    } else if (warp == 9) {
        // ---------------------------------------------------------------------------- MMA issuer
        if (lane == 0 && nblk > 0) {
            constexpr uint32_t idesc_s = instr_desc(BQ, BKV, 0, 0);          // S = Q K^T: both K-major
            constexpr uint32_t idesc_o = instr_desc(BQ, DV, 0, 1);           // O = P V: P K-major, V MN-major
            bool ok = mbar_wait(q_full, 0, A.status);
            int it = 0;
            auto issue_s = [&](int j) {
                const int s = j & 1, m = MAPS == 1 ? 0 : j / nblk;
                for (int kb = 0; kb < KT; ++kb, ++it) {
                    const int slot = it % NK;
                    if (!mbar_wait(&k_full[slot], (uint32_t)((it / NK) & 1), A.status)) return false;
                    tc_fence_after();
                    const uint32_t a0 = smem_u32(sq + (m * KT + kb) * SUB), b0 = smem_u32(sk + slot * SUB);
#pragma unroll
                    for (int k = 0; k < 4; ++k)
                        umma_bf16(tmem_base + TM_S + (uint32_t)(s * BKV), smem_desc(a0 + k * 32, 16, 1024), smem_desc(b0 + k * 32, 16, 1024), idesc_s,
                                  (kb > 0 || k > 0) ? 1u : 0u);
                    umma_commit(&k_empty[slot]);
                }
                umma_commit(&s_full[s]);
                return true;
            };
            if (ok) ok = issue_s(0);
            if (ok && total > 1) ok = issue_s(1);
            for (int j = 0; j < total && ok; ++j) {
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
                if (j + 2 < total) ok = issue_s(j + 2);
            }
            if (!ok) *abort_flag = 1;
        }
    } else {
        // ---------------------------------------------------------------------------- softmax warps
        const int row = 32 * (warp & 3) + lane;          // query row inside the tile = tensor-memory lane
        const int hf = warp >> 2;                        // which page of a block, which DV / 2 columns of O
        const uint32_t lane_addr = tmem_base + ((uint32_t)(32 * (warp & 3)) << 16);
        const int q_pos = T.y + row, q_low = low_of(q_pos, A.window, A.chunked), last_low = low_of(T.y + T.z - 1, A.window, A.chunked);
        float o_acc[DV / 2];
#pragma unroll
        for (int i = 0; i < DV / 2; ++i) o_acc[i] = 0.f;
        float m_run = -INFINITY, l_part = 0.f, alpha_prev = 1.f, l_first = 0.f;
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
        for (int j = 0; j < total; ++j) {
            const int s = j & 1, e = 2 * (MAPS == 1 ? j : j % nblk) + hf;
            const bool turn = MAPS == 2 && j == nblk;    // the first map is complete once O_{j-1} has been added
            const bool there = page_id(e) >= 0;
            if (ok && !*abort_flag) ok = mbar_wait(&s_full[s], (uint32_t)((j >> 1) & 1), A.status);
            else ok = false;
            tc_fence_after();
            float sc[64];
            {
                uint32_t r[32];
                tmem_ld32(lane_addr + TM_S + (uint32_t)(s * BKV + hf * 64), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) sc[i] = __uint_as_float(r[i]) * P.scale_log2;
                tmem_ld32(lane_addr + TM_S + (uint32_t)(s * BKV + hf * 64 + 32), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) sc[32 + i] = __uint_as_float(r[i]) * P.scale_log2;
            }
            const int key0 = pg.at(e) * WA_PAGE;
            if (A.rel) {
                const int far = A.rel_n - 1, d0 = q_pos - key0;
                if (T.y - (key0 + 63) >= far) {          // all keys of the page lie beyond the table for every row of the tile
                    const float b = rel[far];
#pragma unroll
                    for (int i = 0; i < 64; ++i) sc[i] += b;
                } else {
#pragma unroll
                    for (int i = 0; i < 64; ++i) sc[i] += rel[min(max(d0 - i, 0), far)];
                }
            }
            // some row of the tile does not see all 64 keys: one lies ahead of it, or below its lowest and not among the kept
            if (!there || key0 + 63 > T.y || (last_low > key0 && key0 + 63 >= A.keep)) {
                const int ahead = there ? q_pos - key0 : -1, behind = q_low - 1 - key0, kept = A.keep - key0;
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
            if (turn) {
                red[hf * BQ + row] = l_part;
                softmax_sync();
                l_first = red[row] + red[BQ + row];
                softmax_sync();
                l_part = 0.f;
                m_run = -INFINITY;
            }
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
                if (turn) {                              // its output, divided by its sum, waits in tensor memory
                    const float f = l_first > 0.f ? 1.f / l_first : 0.f;
#pragma unroll
                    for (int c = 0; c < DV / 64; ++c) {
                        uint32_t r[32];
#pragma unroll
                        for (int i = 0; i < 32; ++i) { r[i] = __float_as_uint(o_acc[c * 32 + i] * f); o_acc[c * 32 + i] = 0.f; }
                        tmem_st32(lane_addr + TM_KEEP + (uint32_t)(hf * (DV / 2) + c * 32), r);
                    }
                    tmem_st_wait();
                }
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
            if (ok) ok = mbar_wait(o_full, (uint32_t)((total - 1) & 1), A.status);
            tc_fence_after();
            add_o(alpha_prev);
        }
        red[hf * BQ + row] = l_part;
        softmax_sync();
        float l = red[row] + red[BQ + row], f = 1.f;
        if constexpr (MAPS == 2) {                       // d = a1 - mix a2 in place of the output row, divided by its root mean square
            const float f2 = l > 0.f ? A.mix / l : 0.f;
            float ss = 0.f;
#pragma unroll
            for (int c = 0; c < DV / 64; ++c) {
                uint32_t r[32];
                tmem_ld32(lane_addr + TM_KEEP + (uint32_t)(hf * (DV / 2) + c * 32), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 32; ++i) {
                    const float d = __uint_as_float(r[i]) - f2 * o_acc[c * 32 + i];
                    o_acc[c * 32 + i] = d;
                    ss += d * d;
                }
            }
            softmax_sync();                              // the totals have been read
            red[hf * BQ + row] = ss;
            softmax_sync();
            f = rsqrtf((red[row] + red[BQ + row]) / (float)A.Dv + A.mix_eps) * A.mix_gain;
        } else {
            if (A.sink) {
                const float s2 = A.sink[h] * WA_LOG2E, M = fmaxf(m_run, s2);
                f = exp2f(m_run - M);
                l = l * f + exp2f(s2 - M);
            }
            f = l > 0.f ? f / l : 0.f;
        }
        if (row < T.z && T.x + row < A.n && ok) {
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

template <int KT, int DV, int MAPS>
static int launch(const Params& p, cudaStream_t st) {
    const PtbWindowAttn& a = p.A;
    const bool flat = a.flat_rows > 0;
    CUtensorMap mq, mk, mr, mv;
    const int box[4] = {64, WA_PAGE, 1, 1};
    if (flat) {
        const long long heads = a.H, rows = a.flat_rows;
        const long long nk[4] = {a.Dp, rows, heads, 1}, sk[3] = {a.k_ld, a.Dp, a.k_ld}, nv[4] = {a.Dvp, rows, heads, 1}, sv[3] = {a.v_row, a.Dvp, a.v_row};
        const int rot = (a.rot_dim + 15) / 16 * 16;
        const long long nr[4] = {rot, rows, 1, 1}, sr[3] = {a.rot_ld, a.rot_ld, a.rot_ld};
        if (ptb_make_tmap_bf16_3d(&mq, a.q, p.k_own * 64 + rot, a.H, a.n, 64, 1, BQ)) return -1;
        if (ptb_make_tmap_bf16_4d(&mk, a.k_pages, nk, sk, box) || ptb_make_tmap_bf16_4d(&mv, a.v_pages, nv, sv, box)) return -1;
        if (rot ? ptb_make_tmap_bf16_4d(&mr, a.k_rot, nr, sr, box) : (mr = mk, 0)) return -1;
    } else {
        const long long row = (long long)a.maps * a.Dp, page = (long long)a.G * WA_PAGE;
        const long long nk[4] = {row, WA_PAGE, a.G, a.n_pages}, sk[3] = {row, WA_PAGE * row, page * row};
        const long long nv[4] = {a.Dvp, WA_PAGE, a.G, a.n_pages}, sv[3] = {a.Dvp, (long long)WA_PAGE * a.Dvp, page * a.Dvp};
        if (ptb_make_tmap_bf16_3d(&mq, a.q, a.Dp, (long long)a.H * a.maps, a.n, 64, 1, BQ)) return -1;
        if (ptb_make_tmap_bf16_4d(&mk, a.k_pages, nk, sk, box) || ptb_make_tmap_bf16_4d(&mv, a.v_pages, nv, sv, box)) return -1;
        mr = mk;
    }
    using S = Sm<KT, DV, MAPS>;
    static bool attr = false;
    if (!attr) {
        PTB_CUDA_OK(cudaFuncSetAttribute(window_tiles_kernel<KT, DV, MAPS>, cudaFuncAttributeMaxDynamicSharedMemorySize, S::MOST));
        attr = true;
    }
    PTB_CUDA_OK(ptb_launch(window_tiles_kernel<KT, DV, MAPS>, dim3(a.H, a.n_tiles), dim3(NTHREADS), (size_t)S::TOTAL + (a.rel ? (size_t)a.rel_n * 4 : 0), st, ptb_pdl_enabled(), mq, mk, mr, mv, p));
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

template <int KT, int MAPS>
static int launch_v(const Params& p, cudaStream_t st) { return p.A.Dvp <= 64 ? launch<KT, 64, MAPS>(p, st) : launch<KT, 128, MAPS>(p, st); }

}  // namespace wa100
}  // namespace ptb

// Query tiles of a prompt pass against the keys they see, bf16; see PtbWindowAttn.  From pages: sizes as stored up to 128, one or two maps.
// Flat (flat_rows > 0, one map): Dp and rot_dim are a head's own and the shared key size, at most 128 and 64; q is [n][H][Dq] with the own
// part in front, padded with zeros to a multiple of 64, and the shared part, padded to a multiple of 16, behind it.
PTB_API int ptb_window_attn_tiles(const PtbWindowAttn* args, cudaStream_t st) {
    using namespace ptb;
    const PtbWindowAttn& a = *args;
    if (a.n <= 0 || a.n_tiles <= 0) return 0;
    const bool flat = a.flat_rows > 0;
    if (a.G <= 0 || a.H % a.G || a.Dp % 16 || a.Dvp % 16 || a.Dp > 128 || a.Dvp > 128 || a.Dv > a.Dvp || a.window < 1 || a.keep < 0 || a.n_tiles > 65535 ||
        a.maps < 1 || a.maps > 2 || (a.maps == 2 && (a.sink || flat)) || (flat && (a.G != a.H || a.rot_dim > 64 || a.k_ld % 8 || a.v_row % 8 || a.rot_ld % 8)) ||
        (!flat && a.v_ld != a.Dvp) || (a.rel && (flat || a.maps > 1 || a.rel_n < 1 || a.rel_n > wa100::MAX_REL))) {
        ptb_set_error("window attention (tcgen05): bad sizes (H %d, G %d, Dp %d, Dvp %d, window %d, keep %d, maps %d, %d tiles)", a.H, a.G, a.Dp, a.Dvp, a.window, a.keep,
                      a.maps, a.n_tiles);
        return -1;
    }
    int dev = 0;
    PTB_CUDA_OK(cudaGetDevice(&dev));
    PTB_CUDA_OK(cudaSetDevice(dev));     // the tensor-map encoder is a driver call: bind the primary context to this thread
    wa100::Params p;
    memset(&p, 0, sizeof(p));
    p.A = a;
    p.scale_log2 = a.scale * WA_LOG2E;
    p.k_own = (a.Dp + 63) / 64;
    const int kt = p.k_own + (flat && a.rot_dim > 0 ? 1 : 0);
    if (a.maps == 2) return kt == 1 ? wa100::launch_v<1, 2>(p, st) : wa100::launch_v<2, 2>(p, st);
    return kt == 1 ? wa100::launch_v<1, 1>(p, st) : kt == 2 ? wa100::launch_v<2, 1>(p, st) : wa100::launch_v<3, 1>(p, st);
}
