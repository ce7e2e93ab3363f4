// The mixed weights of gated attention (gated_prefill.cu) with both products on tcgen05, for layers of up to 16 heads (with 32, a
// thread's scores and weights of all heads no longer fit the registers of eighteen warps, and the mma.sync kernel is faster).
//
// One CTA: NQ queries x a run of 128-key tiles, all heads.  The queries stay in shared memory; keys stream through a TMA ring, 64 of
// their elements at a time.  Eighteen warps:
//   warp 16  TMA producer;
//   warp 17  owns tensor memory and issues the MMAs from one event loop: S^T(c) = K_c Q_c^T for every key/value head c (rows: keys,
//            columns: query-major, then the head's group) into a ring of column blocks that runs ahead into the next tile, and per
//            query the mixing product D = W talk^T;
//   warps 0-15  four groups of four.  A thread owns a key (its tensor-memory lane); for one query at a time it reads the scores of
//            all heads, forms the weights in fp32 and writes them, each as a high and a low bf16 part, into the 128-byte-swizzled
//            row of its key: the A operand of the mixing product.  Then it reads the mixed weights of the query before and stores
//            them.  The groups take turns at the queries.
// Every wait is bounded.
#pragma once

namespace ptb {
namespace gp {

constexpr int T_PER = 5;              // 128-key tiles per CTA
constexpr int T_GROUPS = 4, T_THREADS = T_GROUPS * 128 + 64, T_STAGES = 5, T_KEYS = 128;
constexpr int T_TMA_WARP = T_GROUPS * 4, T_MMA_WARP = T_TMA_WARP + 1;

struct TcParams {
    WeightsParams W;                   // `per`: 128-key tiles per CTA here
    int NU;                            // column blocks of the score ring
    int groups;                        // CTAs along a tile's queries
};

__device__ __forceinline__ void tma_load_3d(void* dst, const CUtensorMap* map, int c0, int c1, int c2, uint64_t* bar) {
    asm volatile(
        "cp.async.bulk.tensor.3d.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1, {%3, %4, %5}], [%2];" ::"r"(smem_u32(dst)),
        "l"(map), "r"(smem_u32(bar)), "r"(c0), "r"(c1), "r"(c2)
        : "memory");
}
__device__ __forceinline__ void tmem_ld4(uint32_t addr, float* r) {
    uint32_t v[4];
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x4.b32 {%0, %1, %2, %3}, [%4];" : "=r"(v[0]), "=r"(v[1]), "=r"(v[2]), "=r"(v[3]) : "r"(addr) : "memory");
#pragma unroll
    for (int i = 0; i < 4; ++i) r[i] = __uint_as_float(v[i]);
}
__device__ __forceinline__ void tmem_ld2(uint32_t addr, float* r) {
    uint32_t v[2];
    asm volatile("tcgen05.ld.sync.aligned.32x32b.x2.b32 {%0, %1}, [%2];" : "=r"(v[0]), "=r"(v[1]) : "r"(addr) : "memory");
    r[0] = __uint_as_float(v[0]); r[1] = __uint_as_float(v[1]);
}
__device__ __forceinline__ void tmem_ld16(uint32_t taddr, uint32_t* r) {
    asm volatile(
        "tcgen05.ld.sync.aligned.32x32b.x16.b32 {%0, %1, %2, %3, %4, %5, %6, %7, %8, %9, %10, %11, %12, %13, %14, %15}, [%16];"
        : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]), "=r"(r[4]), "=r"(r[5]), "=r"(r[6]), "=r"(r[7]), "=r"(r[8]), "=r"(r[9]), "=r"(r[10]),
          "=r"(r[11]), "=r"(r[12]), "=r"(r[13]), "=r"(r[14]), "=r"(r[15])
        : "r"(taddr)
        : "memory");
}

struct TcSmem {
    int k, w, talk, far, bar, total;   // byte offsets behind the queries
    __host__ __device__ TcSmem(int H, int NQ, int chunks, int HP) {
        k = H * NQ * chunks * 128;
        w = k + T_STAGES * 16384;
        talk = w + T_GROUPS * 16384;
        far = talk + HP * 128;
        bar = far + 128;
        total = bar + 256 + 1024;
    }
};

// HP: heads padded to 16; RV: heads per tensor-memory read, a divisor of the group size (4 or 2); NQ: queries per CTA.
template <int HP, int RV, int NQ>
__global__ void __launch_bounds__(T_THREADS, 1)
gated_weights_tc_kernel(const __grid_constant__ CUtensorMap tmQ, const __grid_constant__ CUtensorMap tmK, const __grid_constant__ TcParams TP) {
    using namespace ptb::gemm;
    const WeightsParams& P = TP.W;
    const GatedAttnParams& A = P.A;
    const int H = A.H, G = A.G, R = H / G, N = R * NQ, chunks = (A.Dp + 63) / 64;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    const TcSmem L(H, NQ, chunks, HP);
    uint8_t* sk = smem + L.k;
    uint8_t* sw = smem + L.w;
    uint8_t* st = smem + L.talk;
    float* far_s = reinterpret_cast<float*>(smem + L.far);
    uint64_t* bars = reinterpret_cast<uint64_t*>(smem + L.bar);
    uint64_t* q_full = bars;
    uint64_t* s_full = bars + 1;             // [2] by tile parity
    uint64_t* s_empty = bars + 3;            // [2]
    uint64_t* w_full = bars + 5;             // [T_GROUPS]
    uint64_t* d_full = w_full + T_GROUPS;    // [T_GROUPS]
    uint64_t* k_full = d_full + T_GROUPS;    // [T_STAGES]
    uint64_t* k_empty = k_full + T_STAGES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(k_empty + T_STAGES);
    volatile int* abort_flag = reinterpret_cast<volatile int*>(tmem_slot + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    constexpr uint32_t D_COL = 512 - T_GROUPS * HP;

    // constants: none of them is written by the kernel before
    if (threadIdx.x == 0) {
        mbar_init(q_full, 1);
        for (int i = 0; i < 2; ++i) { mbar_init(&s_full[i], 1); mbar_init(&s_empty[i], T_GROUPS * 4); }
        for (int i = 0; i < T_GROUPS; ++i) { mbar_init(&w_full[i], 4); mbar_init(&d_full[i], 1); }
        for (int s = 0; s < T_STAGES; ++s) { mbar_init(&k_full[s], 1); mbar_init(&k_empty[s], 1); }
        *abort_flag = 0;
        mbar_fence_init();
        prefetch_tmap(&tmQ);
        prefetch_tmap(&tmK);
    }
    if (warp == T_MMA_WARP) {
        tmem_alloc(tmem_slot, 512);
        tmem_relinquish();
    }
    // the mixing matrix as B operand: row = to head, column 8 u + e = from head 4 u + e % 4 (high parts, then low parts of a unit)
    for (int e = threadIdx.x; e < HP * HP / 4; e += T_THREADS) {
        const int to = e / (HP / 4), u = e % (HP / 4);
        float x[4];
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const int from = 4 * u + i;
            x[i] = to < H && from < H ? (A.talk ? A.talk[(size_t)to * H + from] : (to == from ? 1.f : 0.f)) : 0.f;
        }
        const uint32_t a = fa::pack_bf16(x[0], x[1]), b = fa::pack_bf16(x[2], x[3]);
        *reinterpret_cast<uint4*>(st + to * 128 + ((u ^ (to & 7)) * 16)) = make_uint4(a, b, a, b);
    }
    if (threadIdx.x < 32) far_s[threadIdx.x] = threadIdx.x < H ? -LOG2E * A.bias[(size_t)threadIdx.x * A.nb + A.nb - 1] : 0.f;
    fence_proxy_async();
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_launch_dependents();                 // after the allocation
    pdl_wait();
    const Tile T = P.tiles[blockIdx.x];
    const int q0 = blockIdx.y * NQ, nq = min(NQ, T.count - q0);
    const Band band = band_of(T, A.window);
    const int t_lo = blockIdx.z * P.per, t_hi = nq > 0 ? min(t_lo + P.per, (band.blocks + 1) / 2) : 0, nt = max(0, t_hi - t_lo);
    const int* table = A.page_table + (size_t)T.req * A.pt_stride;

    if (warp == T_TMA_WARP) {
        // ------------------------------------------------------------------------ TMA producer
        if (lane == 0 && nt > 0) {
            bool ok = true;
            mbar_expect_tx(q_full, (uint32_t)(H * NQ * chunks * 128));
            for (int c = 0; c < G; ++c)
                for (int ch = 0; ch < chunks; ++ch) tma_load_3d(smem + (size_t)(c * chunks + ch) * N * 128, &tmQ, ch * 64, c * R, T.tok0 + q0, q_full);
            int s = 0, round = 0;
            for (int kt = 0; kt < nt && ok; ++kt) {
                int page[2];
                for (int b = 0; b < 2; ++b) {
                    const int blk = (t_lo + kt) * 2 + b, col = band.k0 / GA_PAGE + blk;
                    page[b] = blk < band.blocks && col < A.pt_stride ? table[col] : 0;
                    if (page[b] < 0 || page[b] >= A.n_pages) {        // its keys count as invisible below
                        if (A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
                        page[b] = 0;
                    }
                }
                for (int c = 0; c < G && ok; ++c)
                    for (int ch = 0; ch < chunks && ok; ++ch) {
                        if (round > 0) ok = mbar_wait(&k_empty[s], (uint32_t)((round - 1) & 1), A.status);
                        if (!ok || *abort_flag) { ok = false; break; }
                        mbar_expect_tx(&k_full[s], 16384);
                        for (int b = 0; b < 2; ++b) tma_load_2d(sk + s * 16384 + b * 8192, &tmK, ch * 64, (page[b] * G + c) * GA_PAGE, &k_full[s]);
                        if (++s == T_STAGES) { s = 0; ++round; }
                    }
            }
            if (!ok) *abort_flag = 1;
        }
    } else if (warp == T_MMA_WARP) {
        // ------------------------------------------------------------------------ MMA issuer
        if (lane == 0 && nt > 0) {
            const uint32_t id_s = instr_desc(128, N, 0, 0), id_m = instr_desc(128, HP, 0, 0);
            bool ok = mbar_wait(q_full, 0, A.status);
            tc_fence_after();
            // next score block, its chunk, tile and key/value head, its columns; key ring position.  The loop of this one thread paces
            // everything, so it keeps running counters instead of dividing.
            int u = 0, ch = 0, u_kt = 0, u_c = 0, slot = 0, s = 0;
            uint32_t s_par = 0, b_off = 0;
            const uint32_t b_step = (uint32_t)(N * 128), k_base = smem_u32(sk), q_base = smem_u32(smem);
            int consumed = 0;                                           // tiles whose scores have been read
            int m_left = nt * nq, m_q = 0;              // mixing products still to issue, next query of the tile
            uint32_t w_par = 0;                                         // bit g: parity of group g's next weights
            const int units = nt * G;
            int free_until = TP.NU;                                     // blocks below this number have columns to go to
            const uint64_t w_desc = smem_desc(smem_u32(sw), 16, 1024), t_desc = smem_desc(smem_u32(st), 16, 1024);
            uint64_t t0 = global_ns();
            uint32_t idle = 0;
            while (ok && (u < units || m_left > 0)) {
                bool progress = false;
                if (m_left > 0 && mbar_test_wait(&w_full[m_q % T_GROUPS], (w_par >> (m_q % T_GROUPS)) & 1u)) {
                    const int g = m_q % T_GROUPS;
                    tc_fence_after();
#pragma unroll
                    for (int k = 0; k < HP / 8; ++k) umma_bf16(tmem + D_COL + (uint32_t)(g * HP), w_desc + (uint64_t)(g * 1024) + 2 * k, t_desc + 2 * k, id_m, k > 0 ? 1u : 0u);
                    umma_commit(&d_full[g]);
                    w_par ^= 1u << g;
                    --m_left;
                    if (++m_q == nq) m_q = 0;
                    progress = true;
                } else if (u < units) {
                    if (consumed < u_kt && mbar_test_wait(&s_empty[consumed & 1], (uint32_t)((consumed >> 1) & 1))) {
                        tc_fence_after();
                        ++consumed;
                        free_until += G;
                        progress = true;
                    }
                    // at most one tile ahead, and the block's columns are free
                    if (u_kt <= consumed + 1 && u < free_until && mbar_test_wait(&k_full[s], s_par)) {
                        tc_fence_after();
                        const uint32_t d = tmem + (uint32_t)(slot * N);
                        const uint64_t da = smem_desc(k_base + s * 16384, 16, 1024), db = smem_desc(q_base + b_off, 16, 1024);
#pragma unroll
                        for (int k = 0; k < 4; ++k) umma_bf16(d, da + 2 * k, db + 2 * k, id_s, (ch > 0 || k > 0) ? 1u : 0u);   // 32 bytes further each
                        umma_commit(&k_empty[s]);
                        if (++s == T_STAGES) { s = 0; s_par ^= 1; }
                        b_off += b_step;
                        if (++ch == chunks) {
                            ch = 0;
                            ++u;
                            if (++slot == TP.NU) slot = 0;
                            if (++u_c == G) {
                                u_c = 0;
                                b_off = 0;
                                umma_commit(&s_full[u_kt & 1]);
                                ++u_kt;
                            }
                        }
                        progress = true;
                    }
                }
                if (progress) { idle = 0; continue; }
                if ((++idle & 1023u) == 0) {
                    if (idle == 1024u) t0 = global_ns();
                    else if (global_ns() - t0 > 2000000000ull || *abort_flag) {
                        if (A.status) atomicExch(A.status, PTB_ERR_MBARRIER_TIMEOUT);
                        ok = false;
                    }
                }
            }
            if (!ok) *abort_flag = 1;
        }
    } else {
        // ------------------------------------------------------------------------ weights
        const int grp = warp >> 2, row = 32 * (warp & 3) + lane;         // key of the tile = tensor-memory lane
        const uint32_t lane_addr = tmem + ((uint32_t)(32 * (warp & 3)) << 16);
        float cf[6];
        const float xs = A.cap > 0.f ? A.scale * A.inv_cap : A.scale, dot_max = 0.4f / fabsf(xs);
        tanh_poly(A, xs, cf);
        __nv_bfloat16* Pt = P.P + ((size_t)blockIdx.x * H * QT + q0) * P.KW;
        uint8_t* wrow = sw + grp * 16384 + row * 128;
        // where a read of RV heads starts: block of its key/value head and place in the group
        int8_t rd_c[HP / RV];
        int8_t rd_r[HP / RV];
#pragma unroll
        for (int i = 0; i < HP / RV; ++i) { rd_c[i] = (int8_t)(i * RV / R); rd_r[i] = (int8_t)(i * RV % R); }
        const size_t h_step = (size_t)QT * P.KW;
        int slot0 = -G;
        bool ok = true;
        int cnt = 0;
        __nv_bfloat16* pending = nullptr;                                // where this thread's mixed weights of the query before go
        uint32_t d[HP / 2];                                              // pairs of mixed weights, bf16
        auto read_mixed = [&]() {                                        // false: gave up
            if (ok && !*abort_flag) ok = mbar_wait(&d_full[grp], (uint32_t)((cnt - 1) & 1), A.status);
            else ok = false;
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) return;
            tc_fence_after();
#pragma unroll
            for (int b = 0; b < HP; b += 16) {
                uint32_t r[16];
                tmem_ld16(lane_addr + D_COL + (uint32_t)(grp * HP + b), r);
                tmem_ld_wait();
#pragma unroll
                for (int i = 0; i < 8; ++i) d[b / 2 + i] = fa::pack_bf16(__uint_as_float(r[2 * i]), __uint_as_float(r[2 * i + 1]));
            }
            tc_fence_before();
        };
        auto store_mixed = [&]() {
            if (!pending || !ok) return;
            uint16_t* o = reinterpret_cast<uint16_t*>(pending);
#pragma unroll
            for (int h = 0; h < HP; h += 2, o += 2 * h_step)
                if (h < H) {                                             // H is even: groups of two or more
                    o[0] = (uint16_t)d[h / 2];
                    o[h_step] = (uint16_t)(d[h / 2] >> 16);
                }
        };
        for (int kt = 0; kt < nt && ok; ++kt) {
            if (!*abort_flag) ok = mbar_wait(&s_full[kt & 1], (uint32_t)((kt >> 1) & 1), A.status);
            else ok = false;
            ok = __all_sync(0xffffffffu, ok);
            if (!ok) break;
            tc_fence_after();
            const int kcol = (t_lo + kt) * T_KEYS + row, key = band.k0 + kcol, col = key / GA_PAGE;
            bool key_ok = kcol < band.blocks * 64 && col < A.pt_stride;
            if (key_ok) {
                const int page = table[col];
                key_ok = page >= 0 && page < A.n_pages;
            }
            slot0 += G;
            while (slot0 >= TP.NU) slot0 -= TP.NU;
            int at_col[HP / RV];
#pragma unroll
            for (int i = 0; i < HP / RV; ++i) {
                int slot = slot0 + rd_c[i];
                while (slot >= TP.NU) slot -= TP.NU;
                at_col[i] = slot * N + rd_r[i];
            }
            if (grp >= nq) {
                __syncwarp();
                if (lane == 0) mbar_arrive(&s_empty[kt & 1]);
            }
            for (int q = grp; q < nq; q += T_GROUPS) {
                float w[HP];
#pragma unroll
                for (int h = 0; h < HP; h += RV) {
                    if (h < H) {
                        const uint32_t at = lane_addr + (uint32_t)(at_col[h / RV] + q * R);
                        if constexpr (RV == 4) tmem_ld4(at, w + h);
                        else tmem_ld2(at, w + h);
                    } else {
#pragma unroll
                        for (int i = 0; i < RV; ++i) w[h + i] = 0.f;
                    }
                }
                tmem_ld_wait();
                if (q + T_GROUPS >= nq) {                                       // this warp has read all it needs of the tile
                    tc_fence_before();
                    __syncwarp();
                    if (lane == 0) mbar_arrive(&s_empty[kt & 1]);
                }
                const int dist = T.pos0 + q0 + q - key;
                const bool seen = key_ok && dist >= 0 && dist < A.window;
                if (__any_sync(0xffffffffu, seen)) {
                    if (A.cap > 0.f) {
                        float mx = 0.f;
#pragma unroll
                        for (int h = 0; h < HP; ++h) mx = fmaxf(mx, fabsf(w[h]));
                        if (__any_sync(0xffffffffu, mx >= dot_max)) {
#pragma unroll
                            for (int h = 0; h < HP; ++h) w[h] = -LOG2E * A.cap * tanh_any(w[h] * xs);
                        } else {
#pragma unroll
                            for (int h = 0; h < HP; ++h) {
                                const float x = w[h], v = x * x;
                                w[h] = x * fmaf(fmaf(fmaf(fmaf(fmaf(cf[5], v, cf[4]), v, cf[3]), v, cf[2]), v, cf[1]), v, cf[0]);
                            }
                        }
                    } else {
#pragma unroll
                        for (int h = 0; h < HP; ++h) w[h] *= cf[0];
                    }
                    if (__all_sync(0xffffffffu, dist >= A.nb - 1)) {
#pragma unroll
                        for (int h = 0; h < HP; ++h) w[h] = sigmoid_ex2(w[h] + far_s[h]);
                    } else {
                        const int bi = min(max(dist, 0), A.nb - 1);
#pragma unroll
                        for (int h = 0; h < HP; ++h) w[h] = sigmoid_ex2(fmaf(-LOG2E, __ldg(A.bias + (size_t)min(h, H - 1) * A.nb + bi), w[h]));
                    }
                    if (!__all_sync(0xffffffffu, seen)) {
#pragma unroll
                        for (int h = 0; h < HP; ++h) w[h] = seen ? w[h] : 0.f;
                    }
                } else {
#pragma unroll
                    for (int h = 0; h < HP; ++h) w[h] = 0.f;
                }
                if (cnt > 0) {
                    read_mixed();
                    if (!ok) break;
                }
#pragma unroll
                for (int u = 0; u < HP / 4; ++u) {
                    uint4 o;
                    o.x = fa::pack_bf16(w[4 * u], w[4 * u + 1]);
                    o.y = fa::pack_bf16(w[4 * u + 2], w[4 * u + 3]);
                    o.z = fa::pack_bf16(w[4 * u] - __uint_as_float(o.x << 16), w[4 * u + 1] - __uint_as_float(o.x & 0xffff0000u));
                    o.w = fa::pack_bf16(w[4 * u + 2] - __uint_as_float(o.y << 16), w[4 * u + 3] - __uint_as_float(o.y & 0xffff0000u));
                    *reinterpret_cast<uint4*>(wrow + ((u ^ (row & 7)) * 16)) = o;
                }
                fence_proxy_async();
                __syncwarp();
                if (lane == 0) mbar_arrive(&w_full[grp]);
                store_mixed();
                pending = kcol < band.blocks * 64 ? Pt + (size_t)q * P.KW + kcol : nullptr;
                ++cnt;
            }
        }
        if (cnt > 0 && ok) {
            read_mixed();
            store_mixed();
        }
        if (!ok) *abort_flag = 1;
    }
    // ---- teardown
    tc_fence_before();
    __syncthreads();
    if (warp == T_MMA_WARP) tmem_dealloc(tmem, 512);
}

template <int HP, int RV, int NQ>
static int launch_tc(const WeightsParams& w, int tiles, int n_rows, cudaStream_t st) {
    const GatedAttnParams& A = w.A;
    const int R = A.H / A.G, N = R * NQ, chunks = (A.Dp + 63) / 64;
    TcParams p;
    p.W = w;
    p.W.per = T_PER;
    p.NU = (512 - T_GROUPS * HP) / N;
    p.groups = QT / NQ;
    CUtensorMap mq, mk;
    if (ptb_make_tmap_bf16_3d(&mq, A.q, A.Dp, A.H, n_rows, 64, R, NQ)) return -1;
    if (ptb_make_tmap_bf16(&mk, A.k_pages, A.Dp, (long long)A.n_pages * A.G * GA_PAGE, A.Dp, 64, 64)) return -1;
    auto kern = gated_weights_tc_kernel<HP, RV, NQ>;
    static bool attr = false;
    if (!attr) {
        PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        attr = true;
    }
    const TcSmem L(A.H, NQ, chunks, HP);
    const int key_tiles = (w.KW + T_KEYS - 1) / T_KEYS;
    PTB_CUDA_OK(ptb_launch(kern, dim3(tiles, p.groups, (key_tiles + T_PER - 1) / T_PER), dim3(T_THREADS), (size_t)L.total, st, ptb_pdl_enabled(), mq, mk, p));
    return 0;
}

// Sizes the tcgen05 kernel takes: whole groups of 2 or 4 heads per tensor-memory read, key vectors of 64 to 128 elements, and a ring
// of score blocks that holds at least one tile.
static bool tc_supported(const GatedAttnParams& A) {
    const int R = A.H / A.G, NQ = 16, N = R * NQ;
    if (A.H > 16 || A.Dp < 64 || A.Dp > 128 || (R != 2 && R % 4) || N > 256) return false;
    return (512 - T_GROUPS * 16) / N >= A.G;
}
static int launch_tc_any(const WeightsParams& w, int tiles, int n_rows, cudaStream_t st) {
    return w.A.H / w.A.G == 2 ? launch_tc<16, 2, 16>(w, tiles, n_rows, st) : launch_tc<16, 4, 16>(w, tiles, n_rows, st);
}

}  // namespace gp
}  // namespace ptb
