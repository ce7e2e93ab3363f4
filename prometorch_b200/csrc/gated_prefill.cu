// Gated attention (gated_attn.cuh) over many query rows of a prompt, bf16.  The head mixing needs all heads' weights of a
// (query, key) pair at once and the value product needs all keys of a query, so the work is two kernels over tiles of 32 queries
// (of one sequence) with the mixed weights between them as a banded bf16 matrix [tile][head][32][KW]:
//   gated_weights_kernel   scores of all heads on the tensor cores (the queries stay in registers, keys come straight from the
//                          pages), soft cap, bias, sigmoid in fp32, then the head mixing as a second tensor-core product: a
//                          weight enters it as the sum of two bf16 values, the mixing matrix is the left operand, so the result
//                          carries 16 bits of the fp32 weight;
//   gated_values_kernel    O = P V with tcgen05: P tiles and value pages by TMA (the page table picks the box), accumulators in
//                          TMEM; the heads of a key/value head share its pages, their rows fill one 128-row tile.
#include "gated_attn.cuh"
#include "flash_attn.cuh"
#include "gemm_sm100.cuh"
#include <algorithm>

int ptb_make_tmap_bf16(CUtensorMap* map, const void* base, long long inner, long long outer, long long ld, int box_inner, int box_outer);
int ptb_make_tmap_bf16_3d(CUtensorMap* map, const void* base, long long n0, long long n1, long long n2, int b0, int b1, int b2);

namespace ptb {
namespace gp {

constexpr int QT = 32;                 // queries per tile
constexpr int KT = 32;                 // keys per step of the weights kernel
constexpr float LOG2E = 1.4426950408889634f;
constexpr int W_THREADS = 256, W_WARPS = 8;

struct Tile { int tok0, pos0, count, req; };       // rows [tok0, tok0 + count) stand at pos0.. of the sequence in page-table row req

struct Band { int k0, blocks; };                   // first key (a multiple of 64) and 64-key blocks a tile sees
__host__ __device__ __forceinline__ Band band_of(const Tile& t, int window) {
    Band b;
    const int lo = t.pos0 - window + 1;
    b.k0 = (lo > 0 ? lo : 0) / 64 * 64;
    b.blocks = (t.pos0 + t.count - b.k0 + 63) / 64;
    return b;
}

// -log2(e) cap tanh(x) = d (cf0 + cf1 d^2 + ...) with x = xs d: the Taylor series of tanh through x^11, whose next term is below 2e-7
// of the value for |x| < 0.4.  Without a cap, cf0 alone.
__device__ __forceinline__ void tanh_poly(const GatedAttnParams& A, float xs, float* cf) {
    const float a[6] = {1.f, -1.f / 3.f, 2.f / 15.f, -17.f / 315.f, 62.f / 2835.f, -1382.f / 155925.f};
    float m = -LOG2E * (A.cap > 0.f ? A.cap : 1.f) * xs;
#pragma unroll
    for (int k = 0; k < 6; ++k) { cf[k] = a[k] * m; m *= xs * xs; }
}

struct WeightsParams {
    GatedAttnParams A;
    const Tile* tiles;
    __nv_bfloat16* P;                  // [tiles][H][32][KW]
    int KW, per;                       // key steps per CTA
};

// One CTA: 16 queries (half a tile) x at most `per` 32-key steps, all heads.  A warp owns "units" of four consecutive heads.
// Weights of a step in shared memory: row (query i, key j), 16-byte chunk per unit = {4 heads' high parts, 4 heads' low parts},
// chunks XOR-swizzled so that both the stores below and ldmatrix spread over the banks.
__device__ __forceinline__ uint32_t w_off(int i, int j, int chunk, int NC) {
    const int key = ((((j >> 3) & 3) << 1) | (j & 1)) ^ (i & 7);
    return (uint32_t)(((i * KT + j) * NC + (chunk ^ (key & (NC - 1)))) * 16);
}

template <int KS, bool KEEP, bool SAMEC, int NK>
__global__ void __launch_bounds__(W_THREADS, 1) gated_weights_kernel(const __grid_constant__ WeightsParams P) {
    constexpr int NC = 2 * NK, NBUF = NC <= 8 ? 2 : 1;
    constexpr int BUF = 16 * KT * NC * 16;
    extern __shared__ __align__(128) unsigned char smem[];
    uint4* talk_f = reinterpret_cast<uint4*>(smem + NBUF * BUF);       // [m-tile][k-step][lane] fragments of the mixing matrix
    const GatedAttnParams& A = P.A;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    const int H = A.H, R = H / A.G, U = (H + 3) / 4, MT = (H + 15) / 16;
    // constants first: none of them is written by the kernel before
    for (int e = threadIdx.x; e < MT * NK * 32 * 4; e += W_THREADS) {
        const int r = e & 3, l = (e >> 2) & 31, s = (e >> 7) % NK, m = (e >> 7) / NK;
        const int to = m * 16 + (l >> 2) + (r & 1) * 8;
        uint32_t v = 0;
        for (int b = 0; b < 2; ++b) {
            const int k = 2 * (l & 3) + b + (r >> 1) * 8;              // 0..15 inside the step: chunk 2s + k / 8, head k % 4
            const int from = (2 * s + k / 8) * 4 + (k & 3);
            float x = 0.f;
            if (to < H && from < H) x = A.talk ? A.talk[(size_t)to * H + from] : (to == from ? 1.f : 0.f);
            const __nv_bfloat16 h = __float2bfloat16_rn(x);
            v |= (uint32_t)*reinterpret_cast<const uint16_t*>(&h) << (16 * b);
        }
        reinterpret_cast<uint32_t*>(talk_f)[e] = v;
    }
    if (U < NC)                                                        // chunks past U
        for (int e = threadIdx.x; e < NBUF * BUF / 16; e += W_THREADS) reinterpret_cast<uint4*>(smem)[e] = make_uint4(0, 0, 0, 0);
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    const Tile T = P.tiles[blockIdx.x];
    const int half = blockIdx.y * 16;
    if (half >= T.count) return;
    const Band band = band_of(T, A.window);
    const int steps = band.blocks * 2, s_lo = blockIdx.z * P.per, s_hi = min(s_lo + P.per, steps);
    if (s_lo >= s_hi) return;
    const int nq = min(16, T.count - half), q_pos = T.pos0 + half;     // queries q_pos .. q_pos + nq - 1
    const int* table = A.page_table + (size_t)T.req * A.pt_stride;
    __nv_bfloat16* Pt = P.P + ((size_t)blockIdx.x * H * QT + half) * P.KW;
    // key groups: with fewer units than warps, several warps share a unit and take different eight-key columns of a step
    int NG = 1;
    while (NG < 4 && U * NG * 2 <= W_WARPS) NG *= 2;
    const int cols = 4 / NG, n_lo = (warp / U) * cols;
    const bool single = U <= W_WARPS;
    const bool active = single ? warp < U * NG : true;
    const int nch = A.Dp / 8, ks_rt = KEEP ? KS : (A.Dp + 31) / 32;
    const __nv_bfloat16* q = (const __nv_bfloat16*)A.q + (size_t)(T.tok0 + half) * H * A.Dp;
    const __nv_bfloat16* kp = (const __nv_bfloat16*)A.k_pages;
    const uint4 zero4 = make_uint4(0, 0, 0, 0);
    float cf[6];
    const float xs = A.cap > 0.f ? A.scale * A.inv_cap : A.scale, dot_max = 0.4f / fabsf(xs);
    tanh_poly(A, xs, cf);
    auto load_q = [&](int h, int row, int ch) {
        return (h < H && row < nq && ch < nch) ? *reinterpret_cast<const uint4*>(q + ((size_t)row * H + h) * A.Dp + ch * 8) : zero4;
    };
    uint4 qa[KEEP ? 4 : 1][KEEP ? KS : 1][2];
    if constexpr (KEEP) {
        if (active)
#pragma unroll
            for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                for (int s = 0; s < KS; ++s) {
                    qa[hd][s][0] = load_q((warp % U) * 4 + hd, g, 4 * s + t);
                    qa[hd][s][1] = load_q((warp % U) * 4 + hd, g + 8, 4 * s + t);
                }
    }
    // the next eight keys are on their way while the weights of the current ones are formed
    uint4 kb[KEEP && SAMEC ? KS : 1];
    auto fetch = [&](int step, int n) {
        if constexpr (KEEP && SAMEC) {
            const int j = band.k0 + step * KT + n * 8 + g, col = j / GA_PAGE;
            const int page = min(max(col < A.pt_stride ? table[col] : 0, 0), A.n_pages - 1);
            const uint4* kr = reinterpret_cast<const uint4*>(kp + (((size_t)page * A.G + (warp % U) * 4 / R) * GA_PAGE + j % GA_PAGE) * A.Dp);
#pragma unroll
            for (int s = 0; s < KS; ++s) kb[s] = 4 * s + t < nch ? kr[4 * s + t] : zero4;
        }
    };
    if (active && s_lo < s_hi) fetch(s_lo, n_lo);
    for (int step = s_lo; step < s_hi; ++step) {
        const int j0 = band.k0 + step * KT;
        unsigned char* buf = smem + (NBUF == 2 ? (step & 1) * BUF : 0);
        // a step no query of this half sees carries zeros
        const bool dead = j0 > q_pos + nq - 1 || j0 + KT - 1 < q_pos - A.window + 1;
        if (dead) {
            if (active && step + 1 < s_hi) fetch(step + 1, n_lo);
        } else {
            const int col = j0 / GA_PAGE;
            int page = col < A.pt_stride ? table[col] : -1;
            if (page < 0 || page >= A.n_pages) {
                if (threadIdx.x == 0 && A.status) atomicExch(A.status, PTB_ERR_BOUNDS);
                page = -1;
            }
            const bool edge = page < 0 || j0 + KT - 1 > q_pos || j0 < q_pos + 15 - A.window + 1 || nq < 16;
            const bool far = q_pos - (j0 + KT - 1) >= A.nb - 1;        // one bias per head
            for (int u = single ? warp % U : warp; active && u < U; u += single ? U : W_WARPS) {
                const float* bias_u = A.bias + (size_t)u * 4 * A.nb;
                const int hd_max = min(3, H - 1 - u * 4);              // heads of the unit: 0 .. hd_max
                float fb[4];
#pragma unroll
                for (int hd = 0; hd < 4; ++hd) fb[hd] = -LOG2E * __ldg(bias_u + (size_t)min(hd, hd_max) * A.nb + A.nb - 1);
                for (int n = n_lo; n < n_lo + cols; ++n) {
                    float acc[4][4];
#pragma unroll
                    for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                        for (int e = 0; e < 4; ++e) acc[hd][e] = 0.f;
                    const int slot = (j0 + n * 8 + g) % GA_PAGE;
                    auto krow = [&](int c) { return reinterpret_cast<const uint4*>(kp + (((size_t)max(page, 0) * A.G + c) * GA_PAGE + slot) * A.Dp); };
                    if constexpr (KEEP && SAMEC) {
#pragma unroll
                        for (int s = 0; s < KS; ++s)
#pragma unroll
                            for (int hd = 0; hd < 4; ++hd) {
                                const uint4 a = qa[hd][s][0], b = qa[hd][s][1];
                                const uint32_t f0[4] = {a.x, b.x, a.y, b.y}, f1[4] = {a.z, b.z, a.w, b.w};
                                fa::mma16816(acc[hd], f0, kb[s].x, kb[s].y);
                                fa::mma16816(acc[hd], f1, kb[s].z, kb[s].w);
                            }
                        if (n + 1 < n_lo + cols) fetch(step, n + 1);
                        else if (step + 1 < s_hi) fetch(step + 1, n_lo);
                    } else {
                        for (int s = 0; s < ks_rt; ++s) {
                            const int ch = 4 * s + t;
                            uint4 kb = zero4;
#pragma unroll
                            for (int hd = 0; hd < 4; ++hd) {
                                const int h = min(u * 4 + hd, H - 1);
                                if (hd == 0 || h / R != (h - 1) / R) kb = ch < nch ? krow(h / R)[ch] : zero4;
                                uint4 a, b;
                                if constexpr (KEEP) {
                                    // `s` runs to KS: select with a compile-time index
                                    a = zero4; b = zero4;
#pragma unroll
                                    for (int x = 0; x < KS; ++x) if (x == s) { a = qa[hd][x][0]; b = qa[hd][x][1]; }
                                } else {
                                    a = load_q(u * 4 + hd, g, ch);
                                    b = load_q(u * 4 + hd, g + 8, ch);
                                }
                                const uint32_t f0[4] = {a.x, b.x, a.y, b.y}, f1[4] = {a.z, b.z, a.w, b.w};
                                fa::mma16816(acc[hd], f0, kb.x, kb.y);
                                fa::mma16816(acc[hd], f1, kb.z, kb.w);
                            }
                        }
                    }
                    // element e: query g + 8 (e / 2), key n * 8 + 2 t + e % 2.  acc becomes -log2(e) times the capped, scaled score:
                    // as a rule every |x| of the warp is small and an odd polynomial in the dot product itself is enough.
                    if (A.cap > 0.f) {
                        float mx = 0.f;
#pragma unroll
                        for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                            for (int e = 0; e < 4; ++e) mx = fmaxf(mx, fabsf(acc[hd][e]));
                        if (__any_sync(0xffffffffu, mx >= dot_max)) {
#pragma unroll
                            for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                                for (int e = 0; e < 4; ++e) acc[hd][e] = -LOG2E * A.cap * tanh_any(acc[hd][e] * xs);
                        } else {
#pragma unroll
                            for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                                for (int e = 0; e < 4; ++e) {
                                    const float d = acc[hd][e], v = d * d;
                                    acc[hd][e] = d * fmaf(fmaf(fmaf(fmaf(fmaf(cf[5], v, cf[4]), v, cf[3]), v, cf[2]), v, cf[1]), v, cf[0]);
                                }
                        }
                    } else {
#pragma unroll
                        for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                            for (int e = 0; e < 4; ++e) acc[hd][e] *= cf[0];
                    }
                    if (far) {
#pragma unroll
                        for (int hd = 0; hd < 4; ++hd)
#pragma unroll
                            for (int e = 0; e < 4; ++e) acc[hd][e] = sigmoid_ex2(acc[hd][e] + fb[hd]);
                    } else {
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const int bi = min(max(q_pos + g + (e >> 1) * 8 - (j0 + n * 8 + 2 * t + (e & 1)), 0), A.nb - 1);
#pragma unroll
                            for (int hd = 0; hd < 4; ++hd)
                                acc[hd][e] = sigmoid_ex2(fmaf(-LOG2E, __ldg(bias_u + (size_t)min(hd, hd_max) * A.nb + bi), acc[hd][e]));
                        }
                    }
                    if (edge) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const int i = g + (e >> 1) * 8, dist = q_pos + i - (j0 + n * 8 + 2 * t + (e & 1));
                            const bool ok = page >= 0 && i < nq && dist >= 0 && dist < A.window;
#pragma unroll
                            for (int hd = 0; hd < 4; ++hd) acc[hd][e] = ok ? acc[hd][e] : 0.f;
                        }
                    }
#pragma unroll
                    for (int hd = 1; hd < 4; ++hd)
                        if (hd > hd_max)
#pragma unroll
                            for (int e = 0; e < 4; ++e) acc[hd][e] = 0.f;
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int i = g + (e >> 1) * 8, j = n * 8 + 2 * t + (e & 1);
                        uint4 o;
                        o.x = fa::pack_bf16(acc[0][e], acc[1][e]);
                        o.y = fa::pack_bf16(acc[2][e], acc[3][e]);
                        o.z = fa::pack_bf16(acc[0][e] - __uint_as_float(o.x << 16), acc[1][e] - __uint_as_float(o.x & 0xffff0000u));
                        o.w = fa::pack_bf16(acc[2][e] - __uint_as_float(o.y << 16), acc[3][e] - __uint_as_float(o.y & 0xffff0000u));
                        *reinterpret_cast<uint4*>(buf + w_off(i, j, u, NC)) = o;
                    }
                }
            }
        }
        __syncthreads();
        // head mixing: D[to][(i, j)] = talk x weights.  Column n = 2a + b of tile y is key 8 a + 2 y + b, so a lane's columns of the
        // four tiles are the eight keys 8 t .. 8 t + 7 of its rows.
        for (int i = warp; i < nq; i += W_WARPS) {
            __nv_bfloat16* row = Pt + (size_t)i * P.KW + step * KT + 8 * t;
            if (dead) {
                for (int h = g; h < H; h += 8) *reinterpret_cast<uint4*>(row + (size_t)h * QT * P.KW) = zero4;
                continue;
            }
            uint32_t bf[NK <= 4 ? 4 : 1][NK <= 4 ? NK : 1][2];
            const int n = lane & 7, mat = lane >> 3;
            auto load_b = [&](int y, int s, uint32_t* r) {             // two k-steps (four chunks) of tile y
                const int j = 8 * (n >> 1) + 2 * y + (n & 1);
                fa::ldsm4(smem_u32(buf) + w_off(i, j, (2 * s + mat) & (NC - 1), NC), r[0], r[1], r[2], r[3]);
            };
            if constexpr (NK <= 4) {
#pragma unroll
                for (int y = 0; y < 4; ++y)
#pragma unroll
                    for (int s = 0; s < NK; s += 2) {
                        uint32_t r[4];
                        load_b(y, s, r);
                        bf[y][s][0] = r[0]; bf[y][s][1] = r[1];
                        if (s + 1 < NK) { bf[y][s + 1 < NK ? s + 1 : s][0] = r[2]; bf[y][s + 1 < NK ? s + 1 : s][1] = r[3]; }
                    }
            }
            for (int m = 0; m < MT; ++m) {
                float d[4][4];
#pragma unroll
                for (int y = 0; y < 4; ++y)
#pragma unroll
                    for (int e = 0; e < 4; ++e) d[y][e] = 0.f;
                if constexpr (NK <= 4) {
#pragma unroll
                    for (int s = 0; s < NK; ++s) {
                        const uint4 a4 = talk_f[(m * NK + s) * 32 + lane];
                        const uint32_t a[4] = {a4.x, a4.y, a4.z, a4.w};
#pragma unroll
                        for (int y = 0; y < 4; ++y) fa::mma16816(d[y], a, bf[y][s][0], bf[y][s][1]);
                    }
                } else {
#pragma unroll 1
                    for (int s = 0; s < NK; s += 2) {
                        const uint4 a4 = talk_f[(m * NK + s) * 32 + lane], b4 = talk_f[(m * NK + s + 1) * 32 + lane];
                        const uint32_t a[4] = {a4.x, a4.y, a4.z, a4.w}, b[4] = {b4.x, b4.y, b4.z, b4.w};
#pragma unroll
                        for (int y = 0; y < 4; ++y) {
                            uint32_t r[4];
                            load_b(y, s, r);
                            fa::mma16816(d[y], a, r[0], r[1]);
                            fa::mma16816(d[y], b, r[2], r[3]);
                        }
                    }
                }
#pragma unroll
                for (int hr = 0; hr < 2; ++hr) {
                    const int h = m * 16 + g + hr * 8;
                    if (h < H)
                        *reinterpret_cast<uint4*>(row + (size_t)h * QT * P.KW) =
                            make_uint4(fa::pack_bf16(d[0][2 * hr], d[0][2 * hr + 1]), fa::pack_bf16(d[1][2 * hr], d[1][2 * hr + 1]),
                                       fa::pack_bf16(d[2][2 * hr], d[2][2 * hr + 1]), fa::pack_bf16(d[3][2 * hr], d[3][2 * hr + 1]));
                }
            }
        }
        if (NBUF == 1) __syncthreads();
    }
}

}  // namespace gp
}  // namespace ptb

#include "gated_weights_sm100.cuh"

namespace ptb {
namespace gp {

// ---------------------------------------------------------------------------------------------- O = P V
constexpr int V_THREADS = 192, V_STAGES = 3;

struct ValuesParams {
    const Tile* tiles;
    const int* page_table;
    __nv_bfloat16* out;                // [n, H * Dv]
    int pt_stride, n_pages, H, G, Dv, window, mblocks;
    int* status;
};

// BN: value columns of the tile (64, 128, 192 or 256).  Two CTAs fit on an SM up to 128 columns.
template <int BN>
struct VSmem {
    static constexpr int A_BYTES = 128 * 128, B_BYTES = BN * 128, STAGE = A_BYTES + B_BYTES;
    static constexpr int BAR = V_STAGES * STAGE, TOTAL = BAR + 128 + 1024;
    static constexpr int COLS = BN <= 64 ? 64 : BN <= 128 ? 128 : 256;
};

template <int BN>
__global__ void __launch_bounds__(V_THREADS) gated_values_kernel(const __grid_constant__ CUtensorMap tmP, const __grid_constant__ CUtensorMap tmV,
                                                                 const __grid_constant__ ValuesParams P) {
    using namespace ptb::gemm;
    using S = VSmem<BN>;
    extern __shared__ uint8_t smem_raw[];
    uint8_t* smem = reinterpret_cast<uint8_t*>((reinterpret_cast<uintptr_t>(smem_raw) + 1023) & ~(uintptr_t)1023);
    uint64_t* full = reinterpret_cast<uint64_t*>(smem + S::BAR);
    uint64_t* empty = full + V_STAGES;
    uint64_t* done = empty + V_STAGES;
    uint32_t* tmem_slot = reinterpret_cast<uint32_t*>(done + 1);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int c = blockIdx.x / P.mblocks, mb = blockIdx.x % P.mblocks, tile = blockIdx.y;
    const int R = P.H / P.G;
    if (threadIdx.x == 0) {
        for (int s = 0; s < V_STAGES; ++s) { mbar_init(&full[s], 1); mbar_init(&empty[s], 1); }
        mbar_init(done, 1);
        mbar_fence_init();
        prefetch_tmap(&tmP);
        prefetch_tmap(&tmV);
    }
    if (warp == 1) {
        tmem_alloc(tmem_slot, S::COLS);
        tmem_relinquish();
    }
    tc_fence_before();
    __syncthreads();
    tc_fence_after();
    const uint32_t tmem = *tmem_slot;
    pdl_launch_dependents();               // after the allocation: a dependent that wants all of TMEM cannot get in first
    pdl_wait();
    const Tile T = P.tiles[tile];
    const Band band = band_of(T, P.window);
    if (warp == 0) {
        if (lane == 0) {
            const int* table = P.page_table + (size_t)T.req * P.pt_stride;
            const int row0 = (tile * P.H + c * R) * QT + mb * 128;
            bool ok = true;
            for (int kb = 0; kb < band.blocks && ok; ++kb) {
                const int s = kb % V_STAGES;
                if (kb >= V_STAGES) ok = mbar_wait(&empty[s], (uint32_t)((kb / V_STAGES - 1) & 1), P.status);
                if (!ok) break;
                const int col = band.k0 / GA_PAGE + kb;
                int page = col < P.pt_stride ? table[col] : 0;
                if (page < 0 || page >= P.n_pages) {               // its weights are zero; read some page of the pool
                    if (P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
                    page = 0;
                }
                uint8_t* sa = smem + s * S::STAGE;
                mbar_expect_tx(&full[s], S::STAGE);
                tma_load_2d(sa, &tmP, kb * 64, row0, &full[s]);
#pragma unroll
                for (int d = 0; d < BN / 64; ++d) tma_load_2d(sa + S::A_BYTES + d * 8192, &tmV, d * 64, (page * P.G + c) * GA_PAGE, &full[s]);
            }
        }
    } else if (warp == 1) {
        if (lane == 0) {
            constexpr uint32_t idesc = instr_desc(128, BN, 0, 1);
            bool ok = true;
            for (int kb = 0; kb < band.blocks && ok; ++kb) {
                const int s = kb % V_STAGES;
                ok = mbar_wait(&full[s], (uint32_t)((kb / V_STAGES) & 1), P.status);
                if (!ok) break;
                tc_fence_after();
                const uint32_t sa = smem_u32(smem + s * S::STAGE), sb = sa + S::A_BYTES;
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    umma_bf16(tmem, smem_desc(sa + k * 32, 16, 1024), smem_desc(sb + k * 2048, 8192, 1024), idesc, (kb > 0 || k > 0) ? 1u : 0u);
                umma_commit(&empty[s]);
            }
            if (ok) umma_commit(done);
        }
    } else {
        const int quarter = warp & 3, r = mb * 4 + quarter;            // TMEM lanes of a warp: the 32 queries of one head
        const bool ok = mbar_wait(done, 0, P.status);
        tc_fence_after();
        __nv_bfloat16* o = P.out + (size_t)(T.tok0 + lane) * P.H * P.Dv + (size_t)(c * R + r) * P.Dv;
        const bool mine = ok && r < R && lane < T.count;
#pragma unroll 1
        for (int d0 = 0; d0 < P.Dv; d0 += 32) {
            uint32_t v[32];
            tmem_ld32(tmem + ((uint32_t)(quarter * 32) << 16) + (uint32_t)d0, v);
            tmem_ld_wait();
            if (!mine) continue;
            if (P.Dv % 8 == 0 && d0 + 32 <= P.Dv) {
#pragma unroll
                for (int e = 0; e < 32; e += 8)
                    *reinterpret_cast<uint4*>(o + d0 + e) =
                        make_uint4(fa::pack_bf16(__uint_as_float(v[e]), __uint_as_float(v[e + 1])), fa::pack_bf16(__uint_as_float(v[e + 2]), __uint_as_float(v[e + 3])),
                                   fa::pack_bf16(__uint_as_float(v[e + 4]), __uint_as_float(v[e + 5])), fa::pack_bf16(__uint_as_float(v[e + 6]), __uint_as_float(v[e + 7])));
            } else {
#pragma unroll
                for (int e = 0; e < 32; ++e) if (d0 + e < P.Dv) o[d0 + e] = __float2bfloat16_rn(__uint_as_float(v[e]));
            }
        }
    }
    tc_fence_before();
    __syncthreads();
    if (warp == 1) tmem_dealloc(tmem, S::COLS);
}

template <int KS, bool KEEP, bool SAMEC, int NK>
static int launch_weights(const WeightsParams& p, int tiles, cudaStream_t st) {
    auto kern = gated_weights_kernel<KS, KEEP, SAMEC, NK>;
    constexpr int NC = 2 * NK, NBUF = NC <= 8 ? 2 : 1;
    const int smem = NBUF * 16 * KT * NC * 16 + ((p.A.H + 15) / 16) * NK * 512;
    static bool attr = false;
    if (!attr) {
        PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, 227 * 1024));
        attr = true;
    }
    PTB_CUDA_OK(ptb_launch(kern, dim3(tiles, 2, (p.KW / KT + p.per - 1) / p.per), dim3(W_THREADS), (size_t)smem, st, ptb_pdl_enabled(), p));
    return 0;
}
template <int KS, bool KEEP, bool SAMEC>
static int launch_weights_nk(const WeightsParams& p, int tiles, cudaStream_t st) {
    const int U = (p.A.H + 3) / 4;
    if (U <= 2) return launch_weights<KS, KEEP, SAMEC, 1>(p, tiles, st);
    if (U <= 4) return launch_weights<KS, KEEP, SAMEC, 2>(p, tiles, st);
    if (U <= 8) return launch_weights<KS, KEEP, SAMEC, 4>(p, tiles, st);
    if constexpr (!KEEP) return launch_weights<KS, KEEP, SAMEC, 8>(p, tiles, st);
    return -1;
}

template <int BN>
static int launch_values(const CUtensorMap& mp, const CUtensorMap& mv, const ValuesParams& p, int tiles, cudaStream_t st) {
    auto kern = gated_values_kernel<BN>;
    static bool attr = false;
    if (!attr) {
        PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, VSmem<BN>::TOTAL));
        attr = true;
    }
    PTB_CUDA_OK(ptb_launch(kern, dim3(p.G * p.mblocks, tiles), dim3(V_THREADS), (size_t)VSmem<BN>::TOTAL, st, ptb_pdl_enabled(), mp, mv, p));
    return 0;
}

}  // namespace gp
}  // namespace ptb

using namespace ptb;

// Whether ptb_gated_attn_tiles takes these sizes (else: ptb_gated_attn_rows).
PTB_API int ptb_gated_tiles_supported(int H, int G, int Dp, int Dvp) {
    return H >= 1 && H <= 64 && G >= 1 && H % G == 0 && Dp % 16 == 0 && Dp <= 256 && Dvp % 16 == 0 && Dvp >= 64 && Dvp <= 256;
}

// Query tiles of a prompt pass, bf16.  tiles: [n_tiles][4] int32 on the device: first row of q / out, its position, rows (<= 32), row
// of the page table; a tile's rows stand at consecutive positions of one sequence whose keys and values are in the pages.
// weights: scratch of n_tiles * H * 32 * KW bf16, KW (a multiple of 64) at least 64 times the most 64-key blocks a tile sees; per: 32-key steps a CTA of the weights kernel takes.
// tensor_cores: 1 takes the tcgen05 weights kernel where it fits, 0 the mma.sync one.
// q [n_rows, H, Dp], out [n_rows, H Dv].
PTB_API int ptb_gated_attn_tiles(const void* q, void* out, int n_rows, const int* tiles, int n_tiles, int H, int G, int Dp, int Dv, int Dvp,
                                 const int* page_table, int pt_stride, int n_pages, const void* k_pages, const void* v_pages, const float* bias,
                                 int nb, const float* talk, int window, float scale, float cap, void* weights, int KW, int per, int tensor_cores, int* status,
                                 cudaStream_t st) {
    if (n_tiles <= 0) return 0;
    if (!ptb_gated_tiles_supported(H, G, Dp, Dvp) || nb < 1 || window < 1 || KW % 64 || per < 1 || n_tiles > 65535) {
        ptb_set_error("gated attention tiles: bad sizes (H %d, G %d, Dp %d, Dvp %d, KW %d, tiles %d)", H, G, Dp, Dvp, KW, n_tiles);
        return -1;
    }
    gp::WeightsParams w;
    memset(&w, 0, sizeof(w));
    w.A.q = q; w.A.page_table = page_table; w.A.k_pages = k_pages; w.A.bias = bias; w.A.talk = talk; w.A.pt_stride = pt_stride; w.A.n_pages = n_pages;
    w.A.H = H; w.A.G = G; w.A.Dp = Dp; w.A.nb = nb; w.A.window = window; w.A.scale = scale; w.A.cap = cap; w.A.inv_cap = cap > 0.f ? 1.f / cap : 0.f;
    w.A.status = status;
    w.tiles = (const gp::Tile*)tiles; w.P = (__nv_bfloat16*)weights; w.KW = KW; w.per = per;
    const int R = H / G, ks = (Dp + 31) / 32;
    const bool same = R % 4 == 0;
    int rc;
    if (tensor_cores && gp::tc_supported(w.A)) rc = gp::launch_tc_any(w, n_tiles, n_rows, st);
    else if (H > 32 || ks > 4) rc = gp::launch_weights_nk<1, false, false>(w, n_tiles, st);
    else if (!same) rc = ks <= 2 ? gp::launch_weights_nk<2, true, false>(w, n_tiles, st) : gp::launch_weights_nk<4, true, false>(w, n_tiles, st);
    else if (ks <= 2) rc = gp::launch_weights_nk<2, true, true>(w, n_tiles, st);
    else if (ks == 3) rc = gp::launch_weights_nk<3, true, true>(w, n_tiles, st);
    else rc = gp::launch_weights_nk<4, true, true>(w, n_tiles, st);
    if (rc) return rc;
    gp::ValuesParams v;
    v.tiles = (const gp::Tile*)tiles; v.page_table = page_table; v.out = (__nv_bfloat16*)out; v.pt_stride = pt_stride; v.n_pages = n_pages;
    v.H = H; v.G = G; v.Dv = Dv; v.window = window; v.mblocks = (R * gp::QT + 127) / 128; v.status = status;
    CUtensorMap mp, mv;
    if (ptb_make_tmap_bf16(&mp, weights, KW, (long long)n_tiles * H * gp::QT, KW, 64, 128)) return -1;
    if (ptb_make_tmap_bf16(&mv, v_pages, Dvp, (long long)n_pages * G * GA_PAGE, Dvp, 64, 64)) return -1;
    if (Dvp <= 64) rc = gp::launch_values<64>(mp, mv, v, n_tiles, st);
    else if (Dvp <= 128) rc = gp::launch_values<128>(mp, mv, v, n_tiles, st);
    else if (Dvp <= 192) rc = gp::launch_values<192>(mp, mv, v, n_tiles, st);
    else rc = gp::launch_values<256>(mp, mv, v, n_tiles, st);
    if (rc) return rc;
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
