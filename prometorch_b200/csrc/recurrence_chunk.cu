// The recurrent layers of recurrence.cuh over prompts in matrix form, bf16 inputs.  A sequence is cut into chunks of 64 tokens.  With G_i
// the product of the decays of the chunk's tokens up to i (per key channel for the delta rule, a power of the head's decay otherwise)
// and S the state before the chunk,
//     o_i = (q_i G_i)^T S + sum_{j<=i} A_ij u_j,     A_ij = q_i . (k_j G_i / G_j)
//     S'  = G_end S + sum_j (k_j G_end / G_j) u_j^T
// where u is v for decay attention.  For the delta rule (1 + B) u = beta (v - (k G)^T S) with B_ij = beta_i k_i . (k_j G_i / G_j) for
// j < i (a unit lower triangular system, the UT transform of delta-rule attention), hence u = U - W S with U = (1 + B)^-1 beta v and
// W = (1 + B)^-1 beta (k G).  Two kernels:
//   delta_chunk_kernel / delta_head_chunk_kernel / ssd_chunk_kernel / decay_chunk_kernel   everything that does not depend on S, all chunks at once, into a
//                        workspace;
//   chunk_state_kernel                        walks a sequence's chunks for a slice of value columns; S stays in registers.
// What passes between them lies in the order of the mma fragments that will read it: a lane's 16 bytes are its four registers of a 16 x 16
// block, so the walk takes an operand with one 16-byte load per lane.
// Quotients of decays are never formed from products that could overflow: across blocks of 16 tokens both factors refer to the block
// border between the two tokens and are at most 1, inside a block the exponent of every pair is taken directly.
// One decay per head: the quotients are numbers per pair of tokens, so they scale products of the bf16 q and k as they are, and the walk
// takes q and k unscaled, with a factor per row for the product with q and for u on its way into the state.
// State-space steps (MODE 3): q and k belong to a group of heads, so a chunk's fragments of q, k and the products q . k are made once per group
// (ssd_chunk_kernel) and only the pairs' factors per head; u is v, exact in bf16, and the step joins A and the factor of u on its way into
// the state.
// Products run on the tensor cores with every fp32 operand split into two bf16 numbers (three products: 16 bits of both operands).
#include "recurrence.cuh"
#include "flash_attn.cuh"
#include <algorithm>

namespace ptb {
namespace rc {

constexpr int CH = 64, THREADS = 256, WARPS = 8;
constexpr float LOG2E = 1.4426950408889634f;
constexpr float MILD = -60.f;          // log2 of what a block of 16 tokens may keep of a channel: both factors of every pair stay finite

// Workspace of one (chunk, head), in fragments of 512 bytes; the high parts of a matrix, then the low parts.
//   W, Q  left operands   [4 row blocks][DT / 16 column blocks]
//   K     right operand   [DT / 16 blocks of key channels][4 blocks of tokens]
//   A     left operand    [4 row blocks][4 column blocks], those above the diagonal unused
//   G     fp32            the decay of the whole chunk per key channel
//   U     fp32            [Dvp / 16 column blocks][4 row blocks][2 halves of 8 columns][lane] the four accumulator registers
// HEAD (one decay per head): Q and K have no low part, G is [chunk's decay, 3 unused, factor of every row of q (64), of u (64)].
template <int DT, bool HEAD = false>
struct Work {
    static constexpr int TILE = CH * DT * 2, ATILE = CH * CH * 2, PARTS = HEAD ? 1 : 2;
    static constexpr int W = 0, Q = 2 * TILE, K = Q + PARTS * TILE, A = K + PARTS * TILE, G = A + 2 * ATILE, U = G + (HEAD ? 1024 : DT * 4);      // byte offsets
    static __host__ __device__ size_t bytes(int Dvp) { return (size_t)U + (size_t)CH * Dvp * 4; }
};

// State-space steps: q and k of every (chunk, group) first, as in Work without low parts, then of every (chunk, head) A and G.
template <int DT>
struct SsdWork {
    static constexpr int Q = 0, K = Work<DT>::TILE, GROUP = 2 * Work<DT>::TILE, A = 0, G = 2 * Work<DT>::ATILE, HEAD = G + 1024;
};

struct Params {
    PtbRecurrence P;
    unsigned char* work;
    unsigned char* shared;             // MODE 3: the part that the heads of a group share
    size_t stride;                     // bytes per (chunk, head)
    int Dvp;                           // value columns rounded up to 32
    int vec, vec_a;                    // 16-byte loads of x rows, of a (or of low)
};

__device__ __forceinline__ void split2(float a, float b, uint32_t& hi, uint32_t& lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(a, b);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(a - f.x, b - f.y);
    hi = *reinterpret_cast<const uint32_t*>(&h);
    lo = *reinterpret_cast<const uint32_t*>(&l);
}
__device__ __forceinline__ float2 unpack(uint32_t v) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v)); }
// d += a b for operands given as high and low parts
__device__ __forceinline__ void mma3(float* d, const uint32_t* ah, const uint32_t* al, uint32_t bh0, uint32_t bh1, uint32_t bl0, uint32_t bl1) {
    fa::mma16816(d, al, bh0, bh1);
    fa::mma16816(d, ah, bl0, bl1);
    fa::mma16816(d, ah, bh0, bh1);
}
// A lane's four registers of a fragment, given as pairs, to the high and the low part.
__device__ __forceinline__ void store_frag(unsigned char* hi, int part, int frag, int lane, const float2* f) {
    uint4 h, l;
    split2(f[0].x, f[0].y, h.x, l.x); split2(f[1].x, f[1].y, h.y, l.y); split2(f[2].x, f[2].y, h.z, l.z); split2(f[3].x, f[3].y, h.w, l.w);
    unsigned char* p = hi + ((size_t)frag * 32 + lane) * 16;
    *reinterpret_cast<uint4*>(p) = h;
    *reinterpret_cast<uint4*>(p + part) = l;
}
// Columns col, col + 1 (col even) of row r of a high and a low tile in shared memory.
template <int DT>
__device__ __forceinline__ void store_split(unsigned char* hi, unsigned char* lo, int r, int col, float a, float b) {
    uint32_t h, l;
    split2(a, b, h, l);
    const uint32_t off = fa::tile_off<DT>(r, col >> 3) + (col & 7) * 2;
    *reinterpret_cast<uint32_t*>(hi + off) = h;
    *reinterpret_cast<uint32_t*>(lo + off) = l;
}
// Eight columns at once (col a multiple of eight).
template <int DT>
__device__ __forceinline__ void store_split8(unsigned char* hi, unsigned char* lo, int r, int col, const float* f) {
    uint4 h, l;
    split2(f[0], f[1], h.x, l.x); split2(f[2], f[3], h.y, l.y); split2(f[4], f[5], h.z, l.z); split2(f[6], f[7], h.w, l.w);
    const uint32_t off = fa::tile_off<DT>(r, col >> 3);
    *reinterpret_cast<uint4*>(hi + off) = h;
    *reinterpret_cast<uint4*>(lo + off) = l;
}

// Rows of x (columns col .. col + width) of a chunk on their way into a bf16 tile of `pitch` elements per row, zeros past the rows and
// the width (cp.async where `vec` says that rows are 16-byte aligned; the caller commits and waits).
__device__ __forceinline__ void load_rows(const PtbRecurrence& P, bool vec, int row0, int count, int col, int width, int padded, __nv_bfloat16* dst, int pitch) {
    const __nv_bfloat16* x = (const __nv_bfloat16*)P.x;
    const int ch = padded / 8;
    for (int e = threadIdx.x; e < CH * ch; e += THREADS) {
        const int r = e / ch, c = (e % ch) * 8;
        const bool live = r < count && c < width;
        const __nv_bfloat16* s = x + (size_t)(row0 + (live ? r : 0)) * P.ld + col + (live ? c : 0);
        if (vec) fa::cp_async16(smem_u32(dst + r * pitch + c), s, live);
        else {
            uint4 v = make_uint4(0, 0, 0, 0);
            __nv_bfloat16* b = reinterpret_cast<__nv_bfloat16*>(&v);
            if (live)
                for (int k = 0; k < 8 && c + k < width; ++k) b[k] = s[k];
            *reinterpret_cast<uint4*>(dst + r * pitch + c) = v;
        }
    }
}

// (1 + B)^-1 in place of the strictly lower B [64][PA]: the diagonal blocks by substitution (a lane owns a column), then block row after
// block row.  tmp: 16 x 52 floats.  Starts and ends with all threads together.
template <int PA>
__device__ __forceinline__ void unit_lower_inverse(float* ak, float* tmp) {
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    if (warp < 4) {
        float x[16];
        float* b = ak + warp * 16 * PA + warp * 16;
        if (lane < 16) {
#pragma unroll
            for (int i = 0; i < 16; ++i) {
                float v = i == lane ? 1.f : 0.f;
#pragma unroll
                for (int m = 0; m < i; ++m) v = fmaf(-b[i * PA + m], x[m], v);
                x[i] = v;
            }
        }
        __syncwarp();
        if (lane < 16)
#pragma unroll
            for (int i = 0; i < 16; ++i) b[i * PA + lane] = x[i];
    }
    __syncthreads();
    for (int s = 1; s < 4; ++s) {
        const int i = threadIdx.x >> 4, c = threadIdx.x & 15;
        const float* row = ak + (s * 16 + i) * PA;
        for (int r = 0; r < s; ++r) {
            float v = 0.f;
            for (int m = r * 16; m < s * 16; m += 4) {
                const float4 f = *reinterpret_cast<const float4*>(row + m);
                const float* y = ak + m * PA + r * 16 + c;
                v = fmaf(f.x, y[0], fmaf(f.y, y[PA], fmaf(f.z, y[2 * PA], fmaf(f.w, y[3 * PA], v))));
            }
            tmp[i * 52 + r * 16 + c] = v;
        }
        __syncthreads();
        for (int r = 0; r < s; ++r) {
            float v = 0.f;
#pragma unroll
            for (int m = 0; m < 16; ++m) v = fmaf(row[s * 16 + m], tmp[m * 52 + r * 16 + c], v);
            ak[(s * 16 + i) * PA + r * 16 + c] = -v;
        }
        __syncthreads();
    }
}

// ---------------------------------------------------------------------------------------------- delta rule, one chunk
template <int DT>
struct DeltaSmem {
    static constexpr int PB = DT + 8;                  // pitch of the bf16 tiles
    static constexpr int PG = DT + 8;                  // pitch of the decays (floats)
    static constexpr int PA = CH + 4;                  // pitch of the 64 x 64 matrices (floats)
    static constexpr int K = 0, G = K + CH * PB * 2, E = G + CH * PG * 4, A = E + 4 * DT * 4, TH = A + CH * PA * 4, TL = TH + CH * CH * 2;
    static constexpr int TMP = TL + CH * CH * 2, ROW = TMP + 16 * 52 * 4, Q = ROW + 3 * CH * 4 + 32;      // q, and v once q is done with
    static __host__ __device__ int total(int Dvp) { return Q + CH * (Dvp > DT ? Dvp + 8 : PB) * 2; }
};

template <int DT>
__global__ void __launch_bounds__(THREADS, 2) delta_chunk_kernel(const __grid_constant__ Params W) {
    using S = DeltaSmem<DT>;
    using L = Work<DT>;
    extern __shared__ __align__(128) unsigned char smem[];
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem + S::Q);
    __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem + S::K);
    __nv_bfloat16* v_s = q_s;
    float* G_s = reinterpret_cast<float*>(smem + S::G);            // log2 of the product of decays up to and with a token
    float* E_s = reinterpret_cast<float*>(smem + S::E);            // ... of a whole block of 16
    float* ak = reinterpret_cast<float*>(smem + S::A);             // B, then (1 + B)^-1 in its place
    float* tmp = reinterpret_cast<float*>(smem + S::TMP);          // zeros until the inverse uses it
    const float* zeros = tmp;
    float* qn = reinterpret_cast<float*>(smem + S::ROW);
    float* kn = qn + CH;
    float* bt = kn + CH;
    int* next_unit = reinterpret_cast<int*>(bt + CH);
    int* mild = next_unit + 4;
    const PtbRecurrence& P = W.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, D = P.D, Dv = P.Dv, hk = h / (P.H / P.G), PV = W.Dvp + 8;
    const int4 chunk = reinterpret_cast<const int4*>(P.chunks)[blockIdx.x];
    const int row0 = chunk.x, cnt = chunk.y;
    if (row0 < 0 || cnt < 1 || cnt > CH || row0 + cnt > P.n) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        return;
    }
    unsigned char* out = W.work + ((size_t)blockIdx.x * P.H + h) * W.stride;
    load_rows(P, W.vec, row0, cnt, P.q_col + hk * D, D, DT, q_s, S::PB);
    load_rows(P, W.vec, row0, cnt, P.k_col + hk * D, D, DT, k_s, S::PB);
    __nv_bfloat16* low_s = reinterpret_cast<__nv_bfloat16*>(ak);   // over what the scores use later
    const int rank = P.rank, RP = (rank + 15) / 16 * 16 + 8;
    if (P.low) {
        for (int e = threadIdx.x; e < CH * (RP / 8 - 1); e += THREADS) {
            const int r = e / (RP / 8 - 1), c = (e % (RP / 8 - 1)) * 8;
            const bool live = r < cnt && c < rank;
            fa::cp_async16(smem_u32(low_s + r * RP + c), (const __nv_bfloat16*)P.low + (live ? (size_t)(row0 + r) * P.ld_low + c : 0), live);
        }
    } else if (W.vec_a) {
        for (int e = threadIdx.x; e < CH * DT / 4; e += THREADS) {
            const int r = e / (DT / 4), d = e % (DT / 4) * 4;
            const bool live = r < cnt && d < D;
            fa::cp_async16(smem_u32(G_s + r * S::PG + d), (const float*)P.a + (live ? (size_t)(row0 + r) * P.ld_a + h * D + d : 0), live);
        }
    } else
        for (int e = threadIdx.x; e < CH * DT; e += THREADS) {
            const int r = e / DT, d = e % DT;
            G_s[r * S::PG + d] = r < cnt && d < D ? ((const float*)P.a)[(size_t)(row0 + r) * P.ld_a + h * D + d] : 0.f;
        }
    fa::cp_async_commit();
    const float rate = P.decay[h] * LOG2E;
    if (threadIdx.x < CH)
        bt[threadIdx.x] = threadIdx.x < cnt ? sigmoid(__bfloat162float(((const __nv_bfloat16*)P.beta)[(size_t)(row0 + threadIdx.x) * P.ld_beta + h])) : 0.f;
    if (threadIdx.x == 0) *next_unit = WARPS;
    if (threadIdx.x < DT) tmp[threadIdx.x] = 0.f;
    fa::cp_async_wait<0>();
    __syncthreads();
    if (P.low) {                                       // a = low low_w^T: a warp takes 16 channels (and half the rows when there are 4 blocks)
        constexpr int UNITS = DT / 16, SHARE = WARPS / UNITS, RT = 4 / SHARE;
        const int d0 = (warp % UNITS) * 16, rt0 = (warp / UNITS) * RT;
        float c[RT][2][4];
#pragma unroll
        for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int e = 0; e < 8; ++e) c[r][e >> 2][e & 3] = 0.f;
        const __nv_bfloat16* w[2];
        bool live[2];
#pragma unroll
        for (int n = 0; n < 2; ++n) {
            live[n] = d0 + n * 8 + g < D;
            w[n] = (const __nv_bfloat16*)P.low_w + (size_t)(h * D + (live[n] ? d0 + n * 8 + g : 0)) * rank;
        }
#pragma unroll 4
        for (int ks = 0; ks < (rank + 15) / 16; ++ks) {
            uint32_t b[2][2];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int u = 0; u < 2; ++u) {
                    const int k = ks * 16 + 2 * t + 8 * u;         // rank is a multiple of eight
                    b[n][u] = live[n] && k < rank ? *reinterpret_cast<const uint32_t*>(w[n] + k) : 0u;
                }
#pragma unroll
            for (int r = 0; r < RT; ++r) {
                uint32_t a[4];
                fa::ldsm4(smem_u32(low_s + ((rt0 + r) * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * RP + ks * 16 + (lane >> 4) * 8), a[0], a[1], a[2], a[3]);
                fa::mma16816(c[r][0], a, b[0][0], b[0][1]);
                fa::mma16816(c[r][1], a, b[1][0], b[1][1]);
            }
        }
#pragma unroll
        for (int r = 0; r < RT; ++r)
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e)
                    *reinterpret_cast<float2*>(G_s + ((rt0 + r) * 16 + g + 8 * e) * S::PG + d0 + n * 8 + 2 * t) = make_float2(c[r][n][2 * e], c[r][n][2 * e + 1]);
        __syncthreads();
    }
    for (int e = threadIdx.x; e < CH * S::PA; e += THREADS) ak[e] = 0.f;
    for (int r = warp; r < CH; r += WARPS) {
        float a = 0.f, b = 0.f;
        for (int d = lane * 2; d < DT; d += 64) {
            const float2 x = unpack(*reinterpret_cast<const uint32_t*>(q_s + r * S::PB + d)), y = unpack(*reinterpret_cast<const uint32_t*>(k_s + r * S::PB + d));
            a += x.x * x.x + x.y * x.y;
            b += y.x * y.x + y.y * y.y;
        }
        a = warp_sum(a); b = warp_sum(b);
        if (lane == 0) { qn[r] = rsqrtf(a + UNIT_EPS) * rsqrtf((float)D); kn[r] = rsqrtf(b + UNIT_EPS); }
    }
    for (int e = threadIdx.x; e < 4 * DT; e += THREADS) {          // decays (2^-150 is 0) and their running sums inside the blocks of 16
        const int s = e / DT, d = e % DT;
        const float dt = d < D ? P.dt_bias[h * D + d] : 0.f;
        float acc = 0.f;
#pragma unroll 4
        for (int i = 0; i < 16; ++i) {
            float* p = G_s + (s * 16 + i) * S::PG + d;
            acc += s * 16 + i < cnt && d < D ? fmaxf(-150.f, delta_log_decay(*p, dt, rate)) : 0.f;
            *p = acc;
        }
        E_s[s * DT + d] = acc;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < 3 * DT; e += THREADS) {          // ... and what lies before the block
        const int s = e / DT + 1, d = e % DT;
        float base = 0.f;
        for (int r = 0; r < s; ++r) base += E_s[r * DT + d];
#pragma unroll
        for (int i = 0; i < 16; ++i) G_s[(s * 16 + i) * S::PG + d] += base;
    }
    if (warp >= 4) {                                   // whether a block's decays allow one reference for all its pairs
        float least = 0.f;
        for (int d = lane; d < DT; d += 32) least = fminf(least, E_s[(warp - 4) * DT + d]);
        least = -warp_max(-least);
        if (lane == 0) mild[warp - 4] = least > MILD;
    }
    __syncthreads();
    // ---- q G, k G_end / G and G_end
    const float* Ge = G_s + (CH - 1) * S::PG;
    for (int f = warp; f < DT / 4; f += WARPS) {
        const int rb = f / (DT / 16), ks = f % (DT / 16), dp = f >> 2, kt = f & 3;
        float2 x[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) {                  // row g + 8 (u & 1), columns 2t + 8 (u >> 1)
            const int r = rb * 16 + g + 8 * (u & 1), d = ks * 16 + 2 * t + 8 * (u >> 1);
            const float2 q = unpack(*reinterpret_cast<const uint32_t*>(q_s + r * S::PB + d)), G = *reinterpret_cast<const float2*>(G_s + r * S::PG + d);
            x[u] = make_float2(q.x * qn[r] * exp2f(G.x), q.y * qn[r] * exp2f(G.y));
        }
        store_frag(out + L::Q, L::TILE, f, lane, x);
        uint32_t k[4];
        fa::ldsm4_t(smem_u32(k_s + (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::PB + dp * 16 + (lane >> 4) * 8), k[0], k[1], k[2], k[3]);
#pragma unroll
        for (int u = 0; u < 4; ++u) {                  // tokens 2t + 8 (u & 1) and the next, channel g + 8 (u >> 1)
            const int r = kt * 16 + 2 * t + 8 * (u & 1), d = dp * 16 + g + 8 * (u >> 1);
            const float2 v = unpack(k[u]);
            const float E = Ge[d];
            x[u] = make_float2(v.x * kn[r] * exp2f(E - G_s[r * S::PG + d]), v.y * kn[r + 1] * exp2f(E - G_s[(r + 1) * S::PG + d]));
        }
        store_frag(out + L::K, L::TILE, f, lane, x);
    }
    for (int d = threadIdx.x; d < DT; d += THREADS) reinterpret_cast<float*>(out + L::G)[d] = exp2f(Ge[d]);
    // ---- q . k and k . k under the decays: units 0-9 are blocks of 16 x 16 on the tensor cores, six below the diagonal and those on it
    // whose decays are mild; the others 32 pairs each of the remaining blocks on the diagonal
    for (int unit = warp; unit < 10 + 17;) {
        if (unit < 6 || (unit < 10 && mild[unit - 6])) {
            const int s = unit >= 6 ? unit - 6 : unit < 1 ? 1 : unit < 3 ? 2 : 3, r = unit >= 6 ? s : unit - (s == 1 ? 0 : s == 2 ? 1 : 3);
            const float* base = s ? G_s + (s * 16 - 1) * S::PG : zeros;       // both factors refer to the end of the block before s
            float cq[2][4], ck[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) cq[n][e] = ck[n][e] = 0.f;
#pragma unroll 2
            for (int ks = 0; ks < DT / 16; ++ks) {
                uint32_t qh[4], ql[4], kh[4], kl[4];
                float2 b2[2];
#pragma unroll
                for (int u = 0; u < 4; ++u) {                      // row g + 8 (u & 1), columns 2t + 8 (u >> 1)
                    const int i = s * 16 + g + 8 * (u & 1), d = ks * 16 + 2 * t + 8 * (u >> 1);
                    if ((u & 1) == 0) b2[u >> 1] = *reinterpret_cast<const float2*>(base + d);
                    const float2 G = *reinterpret_cast<const float2*>(G_s + i * S::PG + d);
                    const float ex = exp2f(G.x - b2[u >> 1].x), ey = exp2f(G.y - b2[u >> 1].y);
                    const float2 q = unpack(*reinterpret_cast<const uint32_t*>(q_s + i * S::PB + d)), k = unpack(*reinterpret_cast<const uint32_t*>(k_s + i * S::PB + d));
                    split2(q.x * ex, q.y * ey, qh[u], ql[u]);
                    split2(k.x * ex, k.y * ey, kh[u], kl[u]);
                }
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const int j = r * 16 + n * 8 + g;
                    uint32_t bh[2], bl[2];
#pragma unroll
                    for (int u = 0; u < 2; ++u) {
                        const int d = ks * 16 + 2 * t + 8 * u;
                        const float2 G = *reinterpret_cast<const float2*>(G_s + j * S::PG + d);
                        const float2 k = unpack(*reinterpret_cast<const uint32_t*>(k_s + j * S::PB + d));
                        split2(k.x * exp2f(b2[u].x - G.x), k.y * exp2f(b2[u].y - G.y), bh[u], bl[u]);
                    }
                    mma3(cq[n], qh, ql, bh[0], bh[1], bl[0], bl[1]);
                    mma3(ck[n], kh, kl, bh[0], bh[1], bl[0], bl[1]);
                }
            }
            float2 x[4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int i = s * 16 + g + 8 * e, j = r * 16 + n * 8 + 2 * t;
                    const float a = qn[i], b = kn[i] * bt[i], k0 = kn[j], k1 = kn[j + 1];
                    x[n * 2 + e] = make_float2(j <= i ? cq[n][2 * e] * a * k0 : 0.f, j < i ? cq[n][2 * e + 1] * a * k1 : 0.f);
                    *reinterpret_cast<float2*>(ak + i * S::PA + j) = make_float2(j < i ? ck[n][2 * e] * b * k0 : 0.f, j + 1 < i ? ck[n][2 * e + 1] * b * k1 : 0.f);
                }
            store_frag(out + L::A, L::ATILE, s * 4 + r, lane, x);
        } else if (unit >= 10 && !mild[(unit - 10) * 32 / 136] + !mild[((unit - 10) * 32 + 31) / 136]) {
            const int p = (unit - 10) * 32 + lane, s = p / 136, m = p % 136;
            int a = (int)((sqrtf(8.f * m + 1.f) - 1.f) * 0.5f);
            while (a * (a + 1) / 2 > m) --a;
            while ((a + 1) * (a + 2) / 2 <= m) ++a;
            const int i = s * 16 + a, j = s * 16 + m - a * (a + 1) / 2;
            const float* Gi = G_s + i * S::PG;
            const float* Gj = G_s + j * S::PG;
            float sq = 0.f, sk = 0.f;
            for (int d = 0; d < DT; d += 4) {
                const float4 x = *reinterpret_cast<const float4*>(Gi + d), y = *reinterpret_cast<const float4*>(Gj + d);
                const uint2 qr = *reinterpret_cast<const uint2*>(q_s + i * S::PB + d), kr = *reinterpret_cast<const uint2*>(k_s + i * S::PB + d);
                const uint2 jr = *reinterpret_cast<const uint2*>(k_s + j * S::PB + d);
                const float2 q0 = unpack(qr.x), q1 = unpack(qr.y), k0 = unpack(kr.x), k1 = unpack(kr.y), j0 = unpack(jr.x), j1 = unpack(jr.y);
                const float e0 = j0.x * exp2f(x.x - y.x), e1 = j0.y * exp2f(x.y - y.y), e2 = j1.x * exp2f(x.z - y.z), e3 = j1.y * exp2f(x.w - y.w);
                sq = fmaf(q0.x, e0, fmaf(q0.y, e1, fmaf(q1.x, e2, fmaf(q1.y, e3, sq))));
                sk = fmaf(k0.x, e0, fmaf(k0.y, e1, fmaf(k1.x, e2, fmaf(k1.y, e3, sk))));
            }
            const float f = sq * qn[i] * kn[j];
            const __nv_bfloat16 hi = __float2bfloat16_rn(f);
            auto put = [&](int a, int b, __nv_bfloat16 x, __nv_bfloat16 y) {       // element (a, b) of the block, high and low part
                unsigned char* p = out + L::A + (s * 5 * 32 + (a & 7) * 4 + ((b & 7) >> 1)) * 16 + ((a >> 3) + 2 * (b >> 3)) * 4 + (b & 1) * 2;
                *reinterpret_cast<__nv_bfloat16*>(p) = x;
                *reinterpret_cast<__nv_bfloat16*>(p + L::ATILE) = y;
            };
            if (!mild[s]) {
                put(i & 15, j & 15, hi, __float2bfloat16_rn(f - __bfloat162float(hi)));
                if (i != j) {
                    ak[i * S::PA + j] = sk * kn[i] * kn[j] * bt[i];
                    put(j & 15, i & 15, __float2bfloat16_rn(0.f), __float2bfloat16_rn(0.f));
                }
            }
        }
        if (lane == 0) unit = atomicAdd(next_unit, 1);
        unit = __shfl_sync(0xffffffffu, unit, 0);
    }
    __syncthreads();
    load_rows(P, W.vec, row0, cnt, P.v_col + h * Dv, Dv, W.Dvp, v_s, PV);      // over q
    fa::cp_async_commit();
    unit_lower_inverse<S::PA>(ak, tmp);
    for (int e = threadIdx.x; e < CH * CH / 8; e += THREADS) {     // times beta, split
        const int r = e / 8, c = (e % 8) * 8;
        float f[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) f[k] = c + k <= r ? ak[r * S::PA + c + k] * bt[c + k] : 0.f;
        store_split8<CH>(smem + S::TH, smem + S::TL, r, c, f);
    }
    fa::cp_async_wait<0>();
    __syncthreads();
    // ---- W and U: units of 16 columns
    const uint32_t th = smem_u32(smem + S::TH), tl = smem_u32(smem + S::TL);
    for (int unit = warp; unit < DT / 16 + W.Dvp / 16; unit += WARPS) {
        const bool is_w = unit < DT / 16;
        const int n0 = (is_w ? unit : unit - DT / 16) * 16;
        uint32_t bh[4][4], bl[4][4];
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            const __nv_bfloat16* p = is_w ? k_s + n0 : v_s + n0;
            const int pitch = is_w ? S::PB : PV;
            fa::ldsm4_t(smem_u32(p + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * pitch + (lane >> 4) * 8), bh[ks][0], bh[ks][1], bh[ks][2], bh[ks][3]);
        }
        if (is_w)
#pragma unroll
            for (int ks = 0; ks < 4; ++ks)
#pragma unroll
                for (int u = 0; u < 4; ++u) {          // n-block u >> 1, rows 2t, 2t + 1 (+ 8 for odd u)
                    const int j = ks * 16 + 2 * t + 8 * (u & 1), d = n0 + g + 8 * (u >> 1);
                    const float2 k = unpack(bh[ks][u]);
                    split2(k.x * kn[j] * exp2f(G_s[j * S::PG + d]), k.y * kn[j + 1] * exp2f(G_s[(j + 1) * S::PG + d]), bh[ks][u], bl[ks][u]);
                }
#pragma unroll
        for (int rb = 0; rb < 4; ++rb) {
            float c[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) c[n][e] = 0.f;
#pragma unroll
            for (int ks = 0; ks <= rb; ++ks) {
                uint32_t ah[4], al[4];
                fa::load_a<CH>(th, rb * 16, ks, ah);
                fa::load_a<CH>(tl, rb * 16, ks, al);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    if (is_w) mma3(c[n], ah, al, bh[ks][2 * n], bh[ks][2 * n + 1], bl[ks][2 * n], bl[ks][2 * n + 1]);
                    else {
                        fa::mma16816(c[n], al, bh[ks][2 * n], bh[ks][2 * n + 1]);
                        fa::mma16816(c[n], ah, bh[ks][2 * n], bh[ks][2 * n + 1]);
                    }
                }
            }
            if (is_w) {
                const float2 x[4] = {make_float2(c[0][0], c[0][1]), make_float2(c[0][2], c[0][3]), make_float2(c[1][0], c[1][1]), make_float2(c[1][2], c[1][3])};
                store_frag(out + L::W, L::TILE, rb * (DT / 16) + n0 / 16, lane, x);
            } else {
                float4* u = reinterpret_cast<float4*>(out + L::U) + ((n0 / 16) * 4 + rb) * 64 + lane;
                u[0] = make_float4(c[0][0], c[0][1], c[0][2], c[0][3]);
                u[32] = make_float4(c[1][0], c[1][1], c[1][2], c[1][3]);
            }
        }
    }
}

// ---------------------------------------------------------------------------------------------- delta rule with one decay per head
template <int DT>
struct HeadSmem {
    static constexpr int PB = DT + 8, PA = CH + 4;     // pitches of the bf16 tiles and of B
    static constexpr int QB = CH * PB * 2 > CH * CH * 4 ? CH * PB * 2 : CH * CH * 4;         // q, and later the operand of W
    static constexpr int K = 0, Q = K + CH * PB * 2, A = Q + QB, TH = A + CH * PA * 4, TL = TH + CH * CH * 2, TMP = TL + CH * CH * 2, ROW = TMP + 16 * 52 * 4;
    static constexpr int V = ROW + 8 * CH * 4;
    static __host__ __device__ int total(int Dvp) { return V + CH * (Dvp + 8) * 2; }
};

template <int DT>
__global__ void __launch_bounds__(THREADS, 2) delta_head_chunk_kernel(const __grid_constant__ Params W) {
    using S = HeadSmem<DT>;
    using L = Work<DT, true>;
    extern __shared__ __align__(128) unsigned char smem[];
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem + S::Q);
    __nv_bfloat16* k_s = reinterpret_cast<__nv_bfloat16*>(smem + S::K);
    __nv_bfloat16* v_s = reinterpret_cast<__nv_bfloat16*>(smem + S::V);
    float* ak = reinterpret_cast<float*>(smem + S::A);
    float* tmp = reinterpret_cast<float*>(smem + S::TMP);
    float* qn = reinterpret_cast<float*>(smem + S::ROW);           // per row: factors that make unit vectors,
    float* kn = qn + CH;
    float* bt = kn + CH;                                           // beta,
    float* up = bt + CH;                                           // log2 of the decays of its block of 16 up to and with it,
    float* rest = up + CH;                                         // and behind it
    float* E = rest + CH;                                          // [4] of whole blocks; sums of four and fewer terms keep all their bits
    const PtbRecurrence& P = W.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, D = P.D, Dv = P.Dv, hk = h / (P.H / P.G), PV = W.Dvp + 8;
    const int4 chunk = reinterpret_cast<const int4*>(P.chunks)[blockIdx.x];
    const int row0 = chunk.x, cnt = chunk.y;
    if (row0 < 0 || cnt < 1 || cnt > CH || row0 + cnt > P.n) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        return;
    }
    unsigned char* out = W.work + ((size_t)blockIdx.x * P.H + h) * W.stride;
    load_rows(P, W.vec, row0, cnt, P.q_col + hk * D, D, DT, q_s, S::PB);
    load_rows(P, W.vec, row0, cnt, P.k_col + hk * D, D, DT, k_s, S::PB);
    fa::cp_async_commit();
    load_rows(P, W.vec, row0, cnt, P.v_col + h * Dv, Dv, W.Dvp, v_s, PV);
    fa::cp_async_commit();
    if (threadIdx.x < CH) {                            // two warps: a block of 16 tokens is half a warp
        const int i = threadIdx.x;
        const size_t r = (size_t)(row0 + (i < cnt ? i : 0));
        bt[i] = i < cnt ? sigmoid(__bfloat162float(((const __nv_bfloat16*)P.beta)[r * P.ld_beta + h])) : 0.f;
        // 2^-150 is 0
        const float d = i < cnt ? fmaxf(-150.f, delta_log_decay(__bfloat162float(((const __nv_bfloat16*)P.a)[r * P.ld_a + h]), P.dt_bias[h], P.decay[h] * LOG2E)) : 0.f;
        float a = d, b = d;
#pragma unroll
        for (int o = 1; o < 16; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, a, o, 16), y = __shfl_down_sync(0xffffffffu, b, o, 16);
            if ((i & 15) >= o) a += x;
            if ((i & 15) + o < 16) b += y;
        }
        const float behind = __shfl_down_sync(0xffffffffu, b, 1, 16);
        up[i] = a;
        rest[i] = (i & 15) == 15 ? 0.f : behind;
        if ((i & 15) == 15) E[i >> 4] = a;
    }
    fa::cp_async_wait<1>();
    __syncthreads();
    for (int r = warp; r < CH; r += WARPS) {
        float a = 0.f, b = 0.f;
        for (int d = lane * 2; d < DT; d += 64) {
            const float2 x = unpack(*reinterpret_cast<const uint32_t*>(q_s + r * S::PB + d)), y = unpack(*reinterpret_cast<const uint32_t*>(k_s + r * S::PB + d));
            a += x.x * x.x + x.y * x.y;
            b += y.x * y.x + y.y * y.y;
        }
        a = warp_sum(a); b = warp_sum(b);
        if (lane == 0) { qn[r] = rsqrtf(a + UNIT_EPS) * rsqrtf((float)D); kn[r] = rsqrtf(b + UNIT_EPS); }
    }
    // ---- q and k as they are, in fragment order
    for (int f = warp; f < DT / 4; f += WARPS) {
        const int rb = f / (DT / 16), ks = f % (DT / 16), dp = f >> 2, kt = f & 3;
        uint32_t x[4];
        fa::ldsm4(smem_u32(q_s + (rb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::PB + ks * 16 + (lane >> 4) * 8), x[0], x[1], x[2], x[3]);
        *reinterpret_cast<uint4*>(out + L::Q + ((size_t)f * 32 + lane) * 16) = make_uint4(x[0], x[1], x[2], x[3]);
        fa::ldsm4_t(smem_u32(k_s + (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::PB + dp * 16 + (lane >> 4) * 8), x[0], x[1], x[2], x[3]);
        *reinterpret_cast<uint4*>(out + L::K + ((size_t)f * 32 + lane) * 16) = make_uint4(x[0], x[1], x[2], x[3]);
    }
    __syncthreads();
    if (threadIdx.x < CH) {
        const int i = threadIdx.x, b = i >> 4;
        float before = 0.f, after = 0.f;
#pragma unroll
        for (int r = 0; r < 4; ++r) { before += r < b ? E[r] : 0.f; after += r > b ? E[r] : 0.f; }
        float* G = reinterpret_cast<float*>(out + L::G);
        G[4 + i] = qn[i] * exp2f(up[i] + before);
        G[4 + CH + i] = kn[i] * exp2f(rest[i] + after);
        if (i == 0) G[0] = exp2f(E[0] + E[1] + E[2] + E[3]);
    }
    // ---- q . k and k . k in blocks of 16 x 16 up to the diagonal, scaled pair by pair
    for (int unit = warp; unit < 10; unit += WARPS) {
        const int s = unit < 1 ? 0 : unit < 3 ? 1 : unit < 6 ? 2 : 3, r = unit - s * (s + 1) / 2;
        float cq[2][4], ck[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) cq[n][e] = ck[n][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DT / 16; ++ks) {
            uint32_t q[4], k[4], b[4];
            const int a_off = (s * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * S::PB + ks * 16 + (lane >> 4) * 8;
            fa::ldsm4(smem_u32(q_s + a_off), q[0], q[1], q[2], q[3]);
            fa::ldsm4(smem_u32(k_s + a_off), k[0], k[1], k[2], k[3]);
            fa::ldsm4(smem_u32(k_s + (r * 16 + (lane & 7) + (lane >> 4) * 8) * S::PB + ks * 16 + ((lane >> 3) & 1) * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                fa::mma16816(cq[n], q, b[2 * n], b[2 * n + 1]);
                fa::mma16816(ck[n], k, b[2 * n], b[2 * n + 1]);
            }
        }
        float mid = 0.f;                               // whole blocks between the two
        for (int m = r + 1; m < s; ++m) mid += E[m];
        float2 x[4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int i = s * 16 + g + 8 * e, j = r * 16 + n * 8 + 2 * t;
                float w[2];
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const float d = s == r ? up[i] - up[j + c] : up[i] + mid + rest[j + c];
                    w[c] = j + c <= i ? exp2f(d) * kn[j + c] : 0.f;
                }
                const float a = qn[i], b = kn[i] * bt[i];
                x[n * 2 + e] = make_float2(cq[n][2 * e] * a * w[0], cq[n][2 * e + 1] * a * w[1]);
                *reinterpret_cast<float2*>(ak + i * S::PA + j) = make_float2(j < i ? ck[n][2 * e] * b * w[0] : 0.f, j + 1 < i ? ck[n][2 * e + 1] * b * w[1] : 0.f);
            }
        store_frag(out + L::A, L::ATILE, s * 4 + r, lane, x);
    }
    __syncthreads();
    unit_lower_inverse<S::PA>(ak, tmp);
    // ---- times beta for U; times the factor of k's row as well, over q, for W
    for (int e = threadIdx.x; e < CH * CH / 8; e += THREADS) {
        const int r = e / 8, c = (e % 8) * 8;
        float f[8], w[8], before = 0.f;
        for (int m = 0; m < c / 16; ++m) before += E[m];
#pragma unroll
        for (int k = 0; k < 8; ++k) {
            f[k] = c + k <= r ? ak[r * S::PA + c + k] * bt[c + k] : 0.f;
            w[k] = f[k] * kn[c + k] * exp2f(up[c + k] + before);
        }
        store_split8<CH>(smem + S::TH, smem + S::TL, r, c, f);
        store_split8<CH>(smem + S::Q, smem + S::Q + CH * CH * 2, r, c, w);
    }
    fa::cp_async_wait<0>();
    __syncthreads();
    for (int unit = warp; unit < DT / 16 + W.Dvp / 16; unit += WARPS) {        // W and U: units of 16 columns
        const bool is_w = unit < DT / 16;
        const int n0 = (is_w ? unit : unit - DT / 16) * 16;
        const uint32_t th = smem_u32(smem + (is_w ? S::Q : S::TH)), tl = th + CH * CH * 2;
        uint32_t b[4][4];
#pragma unroll
        for (int ks = 0; ks < 4; ++ks) {
            const __nv_bfloat16* p = is_w ? k_s + n0 : v_s + n0;
            fa::ldsm4_t(smem_u32(p + (ks * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * (is_w ? S::PB : PV) + (lane >> 4) * 8), b[ks][0], b[ks][1], b[ks][2], b[ks][3]);
        }
#pragma unroll
        for (int rb = 0; rb < 4; ++rb) {
            float c[2][4];
#pragma unroll
            for (int n = 0; n < 2; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) c[n][e] = 0.f;
#pragma unroll
            for (int ks = 0; ks <= rb; ++ks) {
                uint32_t ah[4], al[4];
                fa::load_a<CH>(th, rb * 16, ks, ah);
                fa::load_a<CH>(tl, rb * 16, ks, al);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    fa::mma16816(c[n], al, b[ks][2 * n], b[ks][2 * n + 1]);
                    fa::mma16816(c[n], ah, b[ks][2 * n], b[ks][2 * n + 1]);
                }
            }
            if (is_w) {
                const float2 x[4] = {make_float2(c[0][0], c[0][1]), make_float2(c[0][2], c[0][3]), make_float2(c[1][0], c[1][1]), make_float2(c[1][2], c[1][3])};
                store_frag(out + L::W, L::TILE, rb * (DT / 16) + n0 / 16, lane, x);
            } else {
                float4* u = reinterpret_cast<float4*>(out + L::U) + ((n0 / 16) * 4 + rb) * 64 + lane;
                u[0] = make_float4(c[0][0], c[0][1], c[0][2], c[0][3]);
                u[32] = make_float4(c[1][0], c[1][1], c[1][2], c[1][3]);
            }
        }
    }
}

// ---------------------------------------------------------------------------------------------- state-space steps, one chunk
// One CTA per (chunk, group, share of the group's heads).
constexpr int SSD_HEADS = THREADS / CH;                // heads whose decays are formed at once
template <int DT>
__global__ void __launch_bounds__(THREADS) ssd_chunk_kernel(const __grid_constant__ Params W, int heads) {
    using L = Work<DT>;
    using M = SsdWork<DT>;
    constexpr int PB = DT + 8, UNITS = 10;
    extern __shared__ __align__(128) unsigned char smem[];
    __nv_bfloat16* q_s = reinterpret_cast<__nv_bfloat16*>(smem);
    __nv_bfloat16* k_s = q_s + CH * PB;
    __shared__ __align__(16) float4 qk_s[UNITS][2][32];            // products of the blocks up to the diagonal, a lane's accumulators
    __shared__ float up_s[SSD_HEADS][CH], rest_s[SSD_HEADS][CH], dt_s[SSD_HEADS][CH], E_s[SSD_HEADS][4];
    const PtbRecurrence& P = W.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_launch_dependents();
    const int grp = blockIdx.y, R = P.H / P.G, D = P.D;
    const int4 chunk = reinterpret_cast<const int4*>(P.chunks)[blockIdx.x];
    const int row0 = chunk.x, cnt = chunk.y;
    if (row0 < 0 || cnt < 1 || cnt > CH || row0 + cnt > P.n) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        return;
    }
    load_rows(P, W.vec, row0, cnt, P.q_col + grp * D, D, DT, q_s, PB);
    load_rows(P, W.vec, row0, cnt, P.k_col + grp * D, D, DT, k_s, PB);
    fa::cp_async_commit();
    fa::cp_async_wait<0>();
    __syncthreads();
    if (blockIdx.z == 0) {
        unsigned char* out = W.shared + ((size_t)blockIdx.x * P.G + grp) * M::GROUP;
        for (int f = warp; f < DT / 4; f += WARPS) {
            const int rb = f / (DT / 16), ks = f % (DT / 16), dp = f >> 2, kt = f & 3;
            uint32_t x[4];
            fa::ldsm4(smem_u32(q_s + (rb * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PB + ks * 16 + (lane >> 4) * 8), x[0], x[1], x[2], x[3]);
            *reinterpret_cast<uint4*>(out + M::Q + ((size_t)f * 32 + lane) * 16) = make_uint4(x[0], x[1], x[2], x[3]);
            fa::ldsm4_t(smem_u32(k_s + (kt * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PB + dp * 16 + (lane >> 4) * 8), x[0], x[1], x[2], x[3]);
            *reinterpret_cast<uint4*>(out + M::K + ((size_t)f * 32 + lane) * 16) = make_uint4(x[0], x[1], x[2], x[3]);
        }
    }
    for (int unit = warp; unit < UNITS; unit += WARPS) {
        const int s = unit < 1 ? 0 : unit < 3 ? 1 : unit < 6 ? 2 : 3, r = unit - s * (s + 1) / 2;
        float c[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) c[n][e] = 0.f;
#pragma unroll
        for (int ks = 0; ks < DT / 16; ++ks) {
            uint32_t q[4], b[4];
            fa::ldsm4(smem_u32(q_s + (s * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * PB + ks * 16 + (lane >> 4) * 8), q[0], q[1], q[2], q[3]);
            fa::ldsm4(smem_u32(k_s + (r * 16 + (lane & 7) + (lane >> 4) * 8) * PB + ks * 16 + ((lane >> 3) & 1) * 8), b[0], b[1], b[2], b[3]);
#pragma unroll
            for (int n = 0; n < 2; ++n) fa::mma16816(c[n], q, b[2 * n], b[2 * n + 1]);
        }
#pragma unroll
        for (int n = 0; n < 2; ++n) qk_s[unit][n][lane] = make_float4(c[n][0], c[n][1], c[n][2], c[n][3]);
    }
    const int h0 = blockIdx.z * heads, h1 = min(R, h0 + heads);
    for (int hb = h0; hb < h1; hb += SSD_HEADS) {
        __syncthreads();                               // the products are there; the heads before are done with
        const int mine = threadIdx.x / CH, i = threadIdx.x % CH, live = min(SSD_HEADS, h1 - hb);
        if (mine < live) {
            const int h = grp * R + hb + mine;
            float dt = 0.f;
            if (i < cnt) dt = softplus(__bfloat162float(((const __nv_bfloat16*)P.a)[(size_t)(row0 + i) * P.ld_a + h]) + P.dt_bias[h]);
            const float d = fmaxf(-150.f, -P.decay[h] * LOG2E * dt);           // 2^-150 is 0
            float a = d, b = d;
#pragma unroll
            for (int o = 1; o < 16; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, a, o, 16), y = __shfl_down_sync(0xffffffffu, b, o, 16);
                if ((i & 15) >= o) a += x;
                if ((i & 15) + o < 16) b += y;
            }
            const float behind = __shfl_down_sync(0xffffffffu, b, 1, 16);
            dt_s[mine][i] = dt;
            up_s[mine][i] = a;
            rest_s[mine][i] = (i & 15) == 15 ? 0.f : behind;
            if ((i & 15) == 15) E_s[mine][i >> 4] = a;
        }
        __syncthreads();
        if (mine < live) {
            const int b = i >> 4;
            float before = 0.f, after = 0.f;
#pragma unroll
            for (int r = 0; r < 4; ++r) { before += r < b ? E_s[mine][r] : 0.f; after += r > b ? E_s[mine][r] : 0.f; }
            float* G = reinterpret_cast<float*>(W.work + ((size_t)blockIdx.x * P.H + grp * R + hb + mine) * W.stride + M::G);
            G[4 + i] = exp2f(up_s[mine][i] + before);
            G[4 + CH + i] = dt_s[mine][i] * exp2f(rest_s[mine][i] + after);
            if (i == 0) G[0] = exp2f(E_s[mine][0] + E_s[mine][1] + E_s[mine][2] + E_s[mine][3]);
        }
        for (int u = warp; u < live * UNITS; u += WARPS) {
            const int hl = u / UNITS, unit = u % UNITS, s = unit < 1 ? 0 : unit < 3 ? 1 : unit < 6 ? 2 : 3, r = unit - s * (s + 1) / 2;
            float mid = 0.f;                           // whole blocks between the two
            for (int m = r + 1; m < s; ++m) mid += E_s[hl][m];
            float2 x[4];
#pragma unroll
            for (int n = 0; n < 2; ++n) {
                const float4 c = qk_s[unit][n][lane];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int i2 = s * 16 + g + 8 * e, j = r * 16 + n * 8 + 2 * t;
                    float w[2];
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        const float d = s == r ? up_s[hl][i2] - up_s[hl][j + k] : up_s[hl][i2] + mid + rest_s[hl][j + k];
                        w[k] = j + k <= i2 ? exp2f(d) * dt_s[hl][j + k] : 0.f;
                    }
                    x[n * 2 + e] = make_float2((e ? c.z : c.x) * w[0], (e ? c.w : c.y) * w[1]);
                }
            }
            store_frag(W.work + ((size_t)blockIdx.x * P.H + grp * R + hb + hl) * W.stride + M::A, L::ATILE, s * 4 + r, lane, x);
        }
    }
}

// ---------------------------------------------------------------------------------------------- fixed decay, one chunk
template <int DT>
__global__ void __launch_bounds__(THREADS) decay_chunk_kernel(const __grid_constant__ Params W) {
    using L = Work<DT>;
    extern __shared__ __align__(128) unsigned char smem[];
    __shared__ float pw[CH + 1];                       // powers of the decay
    unsigned char *qh = smem, *ql = smem + L::TILE, *kh = smem + 2 * L::TILE, *kl = smem + 3 * L::TILE;
    const PtbRecurrence& P = W.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, D = P.D;
    const int4 chunk = reinterpret_cast<const int4*>(P.chunks)[blockIdx.x];
    const int row0 = chunk.x, cnt = chunk.y;
    if (row0 < 0 || cnt < 1 || cnt > CH || row0 + cnt > P.n) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        return;
    }
    unsigned char* out = W.work + ((size_t)blockIdx.x * P.H + h) * W.stride;
    if (warp == 0) {                                   // pw[i] = decay^i: by products over the lanes, then one more step for 32 .. 64
        const float a = P.decay[h];
        float p = lane == 0 ? 1.f : a;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) { const float q = __shfl_up_sync(0xffffffffu, p, o); if (lane >= o) p *= q; }
        const float p32 = __shfl_sync(0xffffffffu, p, 31) * a;
        pw[lane] = p;
        pw[32 + lane] = p * p32;
        if (lane == 31) pw[64] = p32 * p32;
    }
    __syncthreads();
    const __nv_bfloat16* x = (const __nv_bfloat16*)P.x;
    for (int e = threadIdx.x; e < CH * DT / 8; e += THREADS) {
        const int r = e / (DT / 8), d = (e % (DT / 8)) * 8;
        float fq[8], fk[8];
#pragma unroll
        for (int k = 0; k < 8; ++k) fq[k] = fk[k] = 0.f;
        if (r < cnt && d < D) {
            const __nv_bfloat16* q = x + (size_t)(row0 + r) * P.ld + P.q_col + h * D + d;
            const __nv_bfloat16* kk = x + (size_t)(row0 + r) * P.ld + P.k_col + h * D + d;
            if (W.vec) {
                const uint4 a = *reinterpret_cast<const uint4*>(q), b = *reinterpret_cast<const uint4*>(kk);
                const uint32_t *ap = reinterpret_cast<const uint32_t*>(&a), *bp = reinterpret_cast<const uint32_t*>(&b);
#pragma unroll
                for (int k = 0; k < 4; ++k) {
                    const float2 f = unpack(ap[k]), s = unpack(bp[k]);
                    fq[2 * k] = f.x; fq[2 * k + 1] = f.y; fk[2 * k] = s.x; fk[2 * k + 1] = s.y;
                }
            } else
                for (int k = 0; k < 8 && d + k < D; ++k) { fq[k] = __bfloat162float(q[k]); fk[k] = __bfloat162float(kk[k]); }
            if (P.silu)
#pragma unroll
                for (int k = 0; k < 8; ++k) { fq[k] = silu(fq[k]); fk[k] = silu(fk[k]); }
        }
        store_split8<DT>(qh, ql, r, d, fq);
        store_split8<DT>(kh, kl, r, d, fk);
    }
    __syncthreads();
    const uint32_t a_h = smem_u32(qh), a_l = smem_u32(ql), b_h = smem_u32(kh), b_l = smem_u32(kl);
    for (int f = warp; f < DT / 4; f += WARPS) {       // q and k times their powers
        const int rb = f / (DT / 16), ks = f % (DT / 16), dp = f >> 2, kt = f & 3;
        uint32_t hi[4], lo[4];
        float2 x[4];
        fa::load_a<DT>(a_h, rb * 16, ks, hi);
        fa::load_a<DT>(a_l, rb * 16, ks, lo);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float2 a = unpack(hi[u]), b = unpack(lo[u]);
            const float p = pw[rb * 16 + g + 8 * (u & 1) + 1];
            x[u] = make_float2((a.x + b.x) * p, (a.y + b.y) * p);
        }
        store_frag(out + L::Q, L::TILE, f, lane, x);
        fa::load_b_t<DT>(b_h, kt * 16, dp * 2, hi);
        fa::load_b_t<DT>(b_l, kt * 16, dp * 2, lo);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const float2 a = unpack(hi[u]), b = unpack(lo[u]);
            const int r = cnt - 1 - (kt * 16 + 2 * t + 8 * (u & 1));
            x[u] = make_float2(r >= 0 ? (a.x + b.x) * pw[r] : 0.f, r >= 1 ? (a.y + b.y) * pw[r - 1] : 0.f);
        }
        store_frag(out + L::K, L::TILE, f, lane, x);
    }
    for (int unit = warp; unit < 16; unit += WARPS) {              // 16 x 16 blocks up to the diagonal
        const int s = unit >> 2, r = unit & 3;
        if (r > s) continue;
        float c[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) c[n][e] = 0.f;
#pragma unroll 2
        for (int ks = 0; ks < DT / 16; ++ks) {
            uint32_t ah[4], al[4], bh[4], bl[4];
            fa::load_a<DT>(a_h, s * 16, ks, ah);
            fa::load_a<DT>(a_l, s * 16, ks, al);
            fa::load_b<DT>(b_h, r * 16, ks, bh);
            fa::load_b<DT>(b_l, r * 16, ks, bl);
            mma3(c[0], ah, al, bh[0], bh[1], bl[0], bl[1]);
            mma3(c[1], ah, al, bh[2], bh[3], bl[2], bl[3]);
        }
        float2 x[4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int i = s * 16 + g + 8 * e, j = r * 16 + n * 8 + 2 * t;
                x[n * 2 + e] = make_float2(j <= i ? c[n][2 * e] * pw[i - j] : 0.f, j + 1 <= i ? c[n][2 * e + 1] * pw[i - j - 1] : 0.f);
            }
        store_frag(out + L::A, L::ATILE, s * 4 + r, lane, x);
    }
    for (int d = threadIdx.x; d < DT; d += THREADS) reinterpret_cast<float*>(out + L::G)[d] = pw[cnt];
}

// ---------------------------------------------------------------------------------------------- the walk over a sequence's chunks
__device__ __forceinline__ uint4 ld_once(const unsigned char* p) {
    uint4 v;
    asm volatile("ld.global.L1::no_allocate.v4.u32 {%0, %1, %2, %3}, [%4];" : "=r"(v.x), "=r"(v.y), "=r"(v.z), "=r"(v.w) : "l"(p));
    return v;
}
__device__ __forceinline__ uint4 lds_frag(const unsigned char* p, int frag, int lane) { return *reinterpret_cast<const uint4*>(p + (frag * 32 + lane) * 16); }
__device__ __forceinline__ void mma_u4(float* d, const uint4& a, uint32_t b0, uint32_t b1) {
    const uint32_t f[4] = {a.x, a.y, a.z, a.w};
    fa::mma16816(d, f, b0, b1);
}

// One CTA per (VS value columns, head, sequence), eight warps.  Of a chunk, warps 0-3 form u (64 rows) and then the new state, warps 4-7
// the read-out; the state lives transposed, [value][key channel], in the accumulators of warps 0-3 and as two bf16 tiles in shared
// memory for the products that read it.  The other operands arrive by bulk copies through three slots, in the order of their use: W and q
// of a chunk, its k and A, W and q of the next, ...
// With one decay per head (MODE 2, 3) u enters the state times its row's factor, from a second pair of tiles.
template <int DT, int VS, int MODE>
struct StateSmem {
    static constexpr bool HEAD = MODE >= 2;
    using L = Work<DT, HEAD>;
    static constexpr int Q_AT = MODE == 3 ? 0 : 2 * L::TILE;       // of q in its slot
    static constexpr int EVEN = Q_AT + L::PARTS * L::TILE, ODD = L::PARTS * L::TILE + 2 * L::ATILE;
    static constexpr int SLOT = EVEN > ODD ? EVEN : ODD, SH = 3 * SLOT, SL = SH + VS * DT * 2;
    static constexpr int UH = SL + VS * DT * 2, UL = UH + VS * CH * 2, FH = HEAD ? UL + VS * CH * 2 : UH, FL = HEAD ? FH + VS * CH * 2 : UL;
    static constexpr int BAR = FL + VS * CH * 2, TOTAL = BAR + 64;
};
template <int DT, int VS, int MODE>
__global__ void __launch_bounds__(THREADS, 1) chunk_state_kernel(const __grid_constant__ Params W) {
    constexpr bool DELTA = MODE == 1 || MODE == 2, HEAD = MODE >= 2, SSD = MODE == 3;
    using L = Work<DT, HEAD>;
    using S = StateSmem<DT, VS, MODE>;
    using M = SsdWork<DT>;
    constexpr int KS = DT / 16, NT = DT / 32, MT = VS / 16, NB = VS / 8;       // state tiles of a warp: MT x NT of 16 x 8
    extern __shared__ __align__(128) unsigned char smem[];
    unsigned char *s_hi = smem + S::SH, *s_lo = smem + S::SL, *u_hi = smem + S::UH, *u_lo = smem + S::UL;
    uint64_t* bar = reinterpret_cast<uint64_t*>(smem + S::BAR);    // one per slot
    const PtbRecurrence& P = W.P;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    if (threadIdx.x == 0) {
        for (int i = 0; i < 3; ++i) mbar_init(&bar[i], 1);
        mbar_fence_init();
    }
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, v0 = blockIdx.x * VS, D = P.D, Dv = P.Dv;
    const Span sp = span_of(P, blockIdx.z);
    if (sp.slot < 0 || sp.count == 0) return;
    const int first = P.first_chunk[blockIdx.z], chunks = (sp.count + CH - 1) / CH;
    if (first < 0 || first + chunks > P.n_chunks) {
        if (threadIdx.x == 0 && P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
        return;
    }
    const bool owner = warp < 4;                       // of the state channels d0 .. d0 + DT / 4
    const int rb = warp & 3, wr = rb * 16, d0 = rb * (DT / 4);
    const uint32_t sh = smem_u32(s_hi), sl = smem_u32(s_lo), uh = smem_u32(u_hi), ul = smem_u32(u_lo);
    float* st = P.state + (((size_t)sp.slot * P.H + h) * D) * Dv;
    auto tiles = [&](int c) { return W.work + ((size_t)(first + c) * P.H + h) * W.stride; };
    auto factors = [&](int c) { return reinterpret_cast<const float*>(tiles(c) + (SSD ? M::G : L::G)); };
    // load 2c: W and q of chunk c, load 2c + 1: its k and A; load i goes to slot i % 3 once load i - 3 has been read
    auto load = [&](int i) {
        const int s = i % 3;
        const unsigned char* src = tiles(i >> 1);
        if constexpr (SSD) {
            const unsigned char* both = W.shared + ((size_t)(first + (i >> 1)) * P.G + h / (P.H / P.G)) * M::GROUP;
            unsigned char* dst = smem + s * S::SLOT;
            mbar_expect_tx(&bar[s], (i & 1) ? S::ODD : S::EVEN);
            bulk_g2s(dst, both + ((i & 1) ? M::K : M::Q), L::TILE, &bar[s]);
            if (i & 1) bulk_g2s(dst + L::TILE, src + M::A, 2 * L::ATILE, &bar[s]);
        } else if (i & 1) {
            constexpr uint32_t bytes = S::ODD;
            mbar_expect_tx(&bar[s], bytes);
            bulk_g2s(smem + s * S::SLOT, src + L::K, bytes, &bar[s]);
        } else {
            constexpr uint32_t bytes = DELTA ? S::EVEN : 2 * L::TILE;
            mbar_expect_tx(&bar[s], bytes);
            bulk_g2s(smem + s * S::SLOT + (DELTA ? 0 : 2 * L::TILE), src + (DELTA ? L::W : L::Q), bytes, &bar[s]);
        }
    };
    if (threadIdx.x == 0)
        for (int i = 0; i < min(3, 2 * chunks); ++i) load(i);
    float X[MT][NT][4];                                // S^T: row v0 + 16 m + g (+ 8), column d0 + 8 n + 2t (+ 1)
    auto each_state = [&](auto f) {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) f(X[m][n][e], v0 + m * 16 + g + 8 * (e >> 1), d0 + n * 8 + 2 * t + (e & 1));
    };
    auto publish = [&]() {
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) store_split<DT>(s_hi, s_lo, m * 16 + g + 8 * e, d0 + n * 8 + 2 * t, X[m][n][2 * e], X[m][n][2 * e + 1]);
    };
    uint4 base[NB];
    float fac[2] = {1.f, 1.f};                         // HEAD: the factors of this thread's rows of u (warps 0-3)
    const bool pairs = (Dv & 1) == 0 && (P.ld & 1) == 0 && (P.v_col & 1) == 0 && ((uintptr_t)P.x & 3) == 0;
    auto fetch_base = [&](int c) {                     // U in accumulator order, or v (two pairs of bf16)
        const int row0 = sp.row0 + c * CH, cnt = min(CH, sp.count - c * CH);
        if constexpr (HEAD) {
            const float* G = factors(c) + 4 + CH + wr + g;
            fac[0] = G[0]; fac[1] = G[8];
        }
#pragma unroll
        for (int n = 0; n < NB; ++n) {
            if constexpr (DELTA) base[n] = ld_once(tiles(c) + L::U + (((v0 / 16 + (n >> 1)) * 4 + rb) * 64 + (n & 1) * 32 + lane) * 16);
            else {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int r = wr + g + 8 * e, v = v0 + n * 8 + 2 * t;
                    uint32_t f = 0;
                    if (r < cnt && v < Dv) {
                        const __nv_bfloat16* x = (const __nv_bfloat16*)P.x + (size_t)(row0 + r) * P.ld + P.v_col + (size_t)h * Dv + v;
                        if (pairs) f = *reinterpret_cast<const uint32_t*>(x);
                        else f = *reinterpret_cast<const uint16_t*>(x) | (v + 1 < Dv ? (uint32_t)*reinterpret_cast<const uint16_t*>(x + 1) << 16 : 0u);
                    }
                    (e ? base[n].y : base[n].x) = f;
                }
            }
        }
    };
    if (owner) {
        fetch_base(0);
        each_state([&](float& x, int v, int d) { x = sp.pos0 > 0 && v < Dv && d < D ? st[(size_t)d * Dv + v] : 0.f; });
        publish();
    }
    __syncthreads();
    const float skip = SSD ? P.skip[h] : 0.f;
    bool ok = true;
    for (int c = 0; c < chunks; ++c) {
        const unsigned char *wq = smem + (2 * c % 3) * S::SLOT, *ka = smem + ((2 * c + 1) % 3) * S::SLOT;
        const int row0 = sp.row0 + c * CH, cnt = min(CH, sp.count - c * CH);
        float acc[NB][4], low[NB][4], ge[NT][2];       // products of the high parts; those with a low part
#pragma unroll
        for (int n = 0; n < NB; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[n][e] = low[n][e] = 0.f;
        float rq[2] = {1.f, 1.f};                      // HEAD: the factors of this thread's rows of q (warps 4-7)
        if constexpr (HEAD) {
            const float* G = factors(c);
            ge[0][0] = G[0];
            if (!owner) { rq[0] = G[4 + wr + g]; rq[1] = G[4 + wr + g + 8]; }
        } else if (owner) {
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                const float2 f = *reinterpret_cast<const float2*>(tiles(c) + L::G + (d0 + n * 8 + 2 * t) * 4);
                ge[n][0] = f.x; ge[n][1] = f.y;
            }
        }
        if (ok) ok = mbar_wait(&bar[2 * c % 3], (uint32_t)((2 * c / 3) & 1), P.status);
        if (DELTA || !owner) {                         // W S (warps 0-3) or (q G) S (warps 4-7): 16 rows each
            const unsigned char* p = wq + (owner ? 0 : S::Q_AT);
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
                const bool low_part = !HEAD || owner;          // q comes as it is
                const uint4 ah = lds_frag(p, rb * KS + ks, lane), al = low_part ? lds_frag(p + L::TILE, rb * KS + ks, lane) : make_uint4(0, 0, 0, 0);
                uint32_t bh[MT][4], bl[MT][4];
#pragma unroll
                for (int n = 0; n < MT; ++n) { fa::load_b<DT>(sh, n * 16, ks, bh[n]); fa::load_b<DT>(sl, n * 16, ks, bl[n]); }
#pragma unroll
                for (int n = 0; n < NB; ++n) mma_u4(acc[n], ah, bh[n / 2][2 * (n & 1)], bh[n / 2][2 * (n & 1) + 1]);
                if (low_part)
#pragma unroll
                    for (int n = 0; n < NB; ++n) mma_u4(low[n], al, bh[n / 2][2 * (n & 1)], bh[n / 2][2 * (n & 1) + 1]);
#pragma unroll
                for (int n = 0; n < NB; ++n) mma_u4(low[n], ah, bl[n / 2][2 * (n & 1)], bl[n / 2][2 * (n & 1) + 1]);
            }
            if (HEAD && !owner)
#pragma unroll
                for (int n = 0; n < NB; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) { acc[n][e] *= rq[e >> 1]; low[n][e] *= rq[e >> 1]; }
        }
        if (owner) {                                   // u^T, split
#pragma unroll
            for (int n = 0; n < NB; ++n) {
                float u[4];
                if constexpr (DELTA) {
                    u[0] = __uint_as_float(base[n].x); u[1] = __uint_as_float(base[n].y); u[2] = __uint_as_float(base[n].z); u[3] = __uint_as_float(base[n].w);
#pragma unroll
                    for (int e = 0; e < 4; ++e) u[e] -= acc[n][e] + low[n][e];
                } else {
                    const float2 a = unpack(base[n].x), b = unpack(base[n].y);
                    u[0] = a.x; u[1] = a.y; u[2] = b.x; u[3] = b.y;
                    if (MODE == 0 && P.silu)
#pragma unroll
                        for (int e = 0; e < 4; ++e) u[e] = silu(u[e]);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int v = n * 8 + 2 * t + (e & 1), r = wr + g + 8 * (e >> 1);
                    const __nv_bfloat16 hi = __float2bfloat16_rn(u[e]);
                    const uint32_t off = fa::tile_off<CH>(v, r >> 3) + (r & 7) * 2;
                    *reinterpret_cast<__nv_bfloat16*>(u_hi + off) = hi;
                    if constexpr (!SSD) *reinterpret_cast<__nv_bfloat16*>(u_lo + off) = __float2bfloat16_rn(u[e] - __bfloat162float(hi));
                    if constexpr (HEAD) {
                        const float f = u[e] * fac[e >> 1];
                        const __nv_bfloat16 fh = __float2bfloat16_rn(f);
                        *reinterpret_cast<__nv_bfloat16*>(smem + S::FH + off) = fh;
                        *reinterpret_cast<__nv_bfloat16*>(smem + S::FL + off) = __float2bfloat16_rn(f - __bfloat162float(fh));
                    }
                }
            }
            if (c + 1 < chunks) fetch_base(c + 1);
        }
        __syncthreads();                               // u is there; W, q and the state tiles have been read
        if (threadIdx.x == 0 && c + 1 < chunks && ok) load(2 * c + 3);
        if (ok) ok = mbar_wait(&bar[(2 * c + 1) % 3], (uint32_t)(((2 * c + 1) / 3) & 1), P.status);
        if (owner) {
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) X[m][n][e] *= HEAD ? ge[0][0] : ge[n][e & 1];
#pragma unroll
            for (int ks = 0; ks < CH / 16; ++ks) {
                uint32_t a[MT][4], b[MT][4];
                uint4 kh[NT / 2], kl[NT / 2];
#pragma unroll
                for (int n = 0; n < NT / 2; ++n) { kh[n] = lds_frag(ka, (d0 / 16 + n) * 4 + ks, lane); if constexpr (!HEAD) kl[n] = lds_frag(ka + L::TILE, (d0 / 16 + n) * 4 + ks, lane); }
#pragma unroll
                for (int m = 0; m < MT; ++m) { fa::load_a<CH>(uh + (S::FH - S::UH), m * 16, ks, a[m]); fa::load_a<CH>(ul + (S::FL - S::UL), m * 16, ks, b[m]); }
#pragma unroll
                for (int k = 0; k < (HEAD ? 2 : 3); ++k)
#pragma unroll
                    for (int m = 0; m < MT; ++m)
#pragma unroll
                        for (int n = 0; n < NT; ++n) {
                            const uint4& w = k == 2 ? kl[n / 2] : kh[n / 2];
                            fa::mma16816(X[m][n], k == 1 ? b[m] : a[m], (n & 1) ? w.z : w.x, (n & 1) ? w.w : w.y);
                        }
            }
            publish();
        } else {
#pragma unroll
            for (int ks = 0; ks < CH / 16; ++ks)
                if (ks <= rb) {
                    const uint4 kh = lds_frag(ka + L::PARTS * L::TILE, rb * 4 + ks, lane), kl = lds_frag(ka + L::PARTS * L::TILE + L::ATILE, rb * 4 + ks, lane);
                    uint32_t bh[MT][4], bl[MT][4];
#pragma unroll
                    for (int n = 0; n < MT; ++n) { fa::load_b<CH>(uh, n * 16, ks, bh[n]); if constexpr (!SSD) fa::load_b<CH>(ul, n * 16, ks, bl[n]); }
#pragma unroll
                    for (int n = 0; n < NB; ++n) mma_u4(acc[n], kh, bh[n / 2][2 * (n & 1)], bh[n / 2][2 * (n & 1) + 1]);
#pragma unroll
                    for (int n = 0; n < NB; ++n) mma_u4(low[n], kl, bh[n / 2][2 * (n & 1)], bh[n / 2][2 * (n & 1) + 1]);
                    if constexpr (!SSD)
#pragma unroll
                        for (int n = 0; n < NB; ++n) mma_u4(low[n], kh, bl[n / 2][2 * (n & 1)], bl[n / 2][2 * (n & 1) + 1]);
                }
#pragma unroll
            for (int n = 0; n < NB; ++n)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int r = wr + g + 8 * e, v = v0 + n * 8 + 2 * t;
                    float* o = P.out + (size_t)(row0 + r) * P.H * Dv + (size_t)h * Dv + v;
                    float x = acc[n][2 * e] + low[n][2 * e], y = acc[n][2 * e + 1] + low[n][2 * e + 1];
                    if constexpr (SSD) {                 // v is still in its tile
                        auto own = [&](int c) { return __bfloat162float(*reinterpret_cast<const __nv_bfloat16*>(u_hi + fa::tile_off<CH>(c, r >> 3) + (r & 7) * 2)); };
                        x = fmaf(skip, own(n * 8 + 2 * t), x);
                        y = fmaf(skip, own(n * 8 + 2 * t + 1), y);
                    }
                    if (r >= cnt) continue;
                    if (v + 1 < Dv && (Dv & 1) == 0) *reinterpret_cast<float2*>(o) = make_float2(x, y);
                    else {
                        if (v < Dv) o[0] = x;
                        if (v + 1 < Dv) o[1] = y;
                    }
                }
        }
        __syncthreads();                               // the new state is there; k, A and u have been read
        if (threadIdx.x == 0 && c + 2 < chunks && ok) load(2 * c + 4);
    }
    if (owner) each_state([&](float& x, int v, int d) { if (ok && v < Dv && d < D) st[(size_t)d * Dv + v] = x; });
}

template <int DT, int VS, int MODE>
static int launch_state(const Params& p, cudaStream_t st) {
    const dim3 grid((p.P.Dv + VS - 1) / VS, p.P.H, p.P.n_seqs);
    constexpr int smem = StateSmem<DT, VS, MODE>::TOTAL;
    PTB_CUDA_OK(cudaFuncSetAttribute(chunk_state_kernel<DT, VS, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
    PTB_CUDA_OK(ptb_launch(chunk_state_kernel<DT, VS, MODE>, grid, dim3(THREADS), (size_t)smem, st, ptb_pdl_enabled(), p));
    return 0;
}
template <int DT, int VS>
static int launch_state(const Params& p, cudaStream_t st) {
    return p.P.delta == 3 ? launch_state<DT, VS, 3>(p, st) : p.P.delta == 2 ? launch_state<DT, VS, 2>(p, st) : p.P.delta ? launch_state<DT, VS, 1>(p, st) : launch_state<DT, VS, 0>(p, st);
}

template <int DT>
static int launch(Params p, cudaStream_t st) {
    const dim3 grid(p.P.n_chunks, p.P.H);
    const bool pdl = ptb_pdl_enabled();
    auto go = [&](auto kern, int smem) {
        PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        PTB_CUDA_OK(ptb_launch(kern, grid, dim3(THREADS), (size_t)smem, st, pdl, p));
        return 0;
    };
    if (p.P.delta == 3) {
        p.shared = p.work;
        p.work += (size_t)p.P.n_chunks * p.P.G * SsdWork<DT>::GROUP;
        const int R = p.P.H / p.P.G;                   // shares of whole batches of heads, about three CTAs per SM
        const long long most = std::max<long long>(1, 444LL / std::max<long long>(1, (long long)p.P.n_chunks * p.P.G));
        const int heads = (int)((R + most - 1) / most + SSD_HEADS - 1) / SSD_HEADS * SSD_HEADS, smem = 2 * CH * (DT + 8) * 2;
        auto kern = ssd_chunk_kernel<DT>;
        PTB_CUDA_OK(cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, smem));
        PTB_CUDA_OK(ptb_launch(kern, dim3(p.P.n_chunks, p.P.G, (R + heads - 1) / heads), dim3(THREADS), (size_t)smem, st, pdl, p, heads));
    } else if (p.P.delta == 2 ? go(delta_head_chunk_kernel<DT>, HeadSmem<DT>::total(p.Dvp))
                       : p.P.delta ? go(delta_chunk_kernel<DT>, DeltaSmem<DT>::total(p.Dvp)) : go(decay_chunk_kernel<DT>, 4 * Work<DT>::TILE)) return -1;
    // few CTAs: narrow slices, so that more of them share the walk
    const long long wide = (long long)((p.P.Dv + 31) / 32) * p.P.H * p.P.n_seqs;
    if (wide <= 74 ? launch_state<DT, 16>(p, st) : launch_state<DT, 32>(p, st)) return -1;
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}

}  // namespace rc

int recurrence_check(const PtbRecurrence& p);

static size_t chunk_bytes(const PtbRecurrence& p) {
    const int Dvp = (p.Dv + 31) / 32 * 32;
    if (p.delta == 3) return rc::SsdWork<64>::HEAD;                // and what a group's heads share
    if (p.delta == 2) return p.D <= 64 ? rc::Work<64, true>::bytes(Dvp) : rc::Work<128, true>::bytes(Dvp);
    return p.D <= 64 ? rc::Work<64>::bytes(Dvp) : rc::Work<128>::bytes(Dvp);
}

}  // namespace ptb

using namespace ptb;

// Bytes of workspace of ptb_recurrence_chunked, or -1 for sizes it does not take (bf16, D and Dv up to 128).
PTB_API long long ptb_recurrence_chunked_bytes(const PtbRecurrence* args) {
    const PtbRecurrence& p = *args;
    if (!p.bf16 || p.D > 128 || p.Dv > 128 || p.n_chunks < 1) return -1;
    const long long shared = p.delta == 3 ? (long long)p.G * (p.D <= 64 ? rc::SsdWork<64>::GROUP : rc::SsdWork<128>::GROUP) : 0;
    return ((long long)chunk_bytes(p) * p.H + shared) * p.n_chunks;
}

// ptb_recurrence for a prompt pass, in chunks of 64 rows; see PtbRecurrence.
PTB_API int ptb_recurrence_chunked(const PtbRecurrence* args, void* work, long long bytes, cudaStream_t st) {
    if (args->n <= 0 || args->n_seqs <= 0) return 0;
    if (recurrence_check(*args)) return -1;
    const long long need = ptb_recurrence_chunked_bytes(args);
    if (need < 0 || bytes < need || !args->seqs || !args->chunks || !args->first_chunk || ((uintptr_t)work & 127)) {
        ptb_set_error("recurrence_chunked: sizes (D %d, Dv %d), workspace (%lld of %lld bytes) or chunk table", args->D, args->Dv, bytes, need);
        return -1;
    }
    rc::Params p;
    p.P = *args;
    p.work = (unsigned char*)work;
    p.shared = nullptr;
    p.stride = chunk_bytes(*args);
    p.Dvp = (args->Dv + 31) / 32 * 32;
    p.vec = args->D % 8 == 0 && args->Dv % 8 == 0 && args->ld % 8 == 0 && args->q_col % 8 == 0 && args->k_col % 8 == 0 && args->v_col % 8 == 0 &&
            ((uintptr_t)args->x & 15) == 0;
    if (args->delta && args->low &&
        (!args->low_w || args->rank < 8 || args->rank > 256 || args->rank % 8 || args->ld_low % 8 || (((uintptr_t)args->low | (uintptr_t)args->low_w) & 15))) {
        ptb_set_error("recurrence_chunked: a low-rank product of rank %d (a multiple of eight up to 256, 16-byte aligned rows)", args->rank);
        return -1;
    }
    p.vec_a = args->D % 4 == 0 && args->ld_a % 4 == 0 && ((uintptr_t)args->a & 15) == 0;
    return args->D <= 64 ? rc::launch<64>(p, st) : rc::launch<128>(p, st);
}
