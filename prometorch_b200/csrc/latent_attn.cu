// Latent attention, the parts around its softmax for few query rows:
//   head_linear_kernel   a matrix per head: folds W_uk into the queries (and appends their rotated part), applies W_uv to weighted latents
//                        (and the gate).  Any size, fp32 arithmetic.
#include "window_attn.cuh"
#include <algorithm>

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

// HL_ROWS rows x HL_COLS outputs of one head per CTA: a warp takes eight outputs, its lanes share K.  The last column block pads and rotates.
template <typename T>
__global__ void __launch_bounds__(HL_THREADS) head_linear_kernel(const __grid_constant__ HeadLinear P) {
    pdl_wait();
    pdl_launch_dependents();
    const int h = blockIdx.y, r0 = blockIdx.z * HL_ROWS, blocks = (P.N + HL_COLS - 1) / HL_COLS, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int rows = min(HL_ROWS, P.n - r0);
    if ((int)blockIdx.x == blocks) {
        for (int e = threadIdx.x; e < rows * (P.os - P.N); e += HL_THREADS) {
            const int r = r0 + e / (P.os - P.N), c = P.N + e % (P.os - P.N), d = c - P.rot_at;
            float v = 0.f;
            if (d >= 0 && d < P.rot) {
                int pos = P.pos[(size_t)r * P.pos_stride];
                if (pos < 0 || pos >= P.positions) {
                    if (P.status) atomicExch(P.status, PTB_ERR_BOUNDS);
                    pos = 0;
                }
                const T* x = (const T*)P.x + (size_t)r * P.ldx + (size_t)h * P.xs + P.K;
                const size_t at = (size_t)pos * (P.rot / 2) + d / 2;
                const float cs = P.cos[at], sn = P.sin[at], a = (float)x[d], b = (float)x[d ^ 1];
                v = (d & 1) ? a * cs + b * sn : a * cs - b * sn;
            }
            ((T*)P.out)[(size_t)r * P.ldo + (size_t)h * P.os + c] = (T)v;
        }
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

}  // namespace la
}  // namespace ptb

using namespace ptb;

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
        if (bf16) PTB_CUDA_OK(ptb_launch(head_linear_kernel<__nv_bfloat16>, grid, dim3(HL_THREADS), 0, st, pdl, p));
        else PTB_CUDA_OK(ptb_launch(head_linear_kernel<float>, grid, dim3(HL_THREADS), 0, st, pdl, p));
    }
    PTB_CUDA_OK(cudaGetLastError());
    return 0;
}
