// Softmax attention inside a sliding window over the paged cache: the query at position p sees the keys p - window + 1 .. p and the
// first `keep` tokens of its sequence.  A sink adds exp(sink_h) to a head's denominator; a gate scales the head's output by its sigmoid.
#pragma once
#include "common.cuh"

namespace ptb {

constexpr int WA_PAGE = 64;
constexpr int WA_KEYS = 128;           // most keys of one CTA of the row kernels
constexpr float WA_LOG2E = 1.4426950408889634f;

struct WindowAttnParams {
    const void* q;                     // [n, H, Dp]
    void* out;                         // [n, H Dv]
    float* work;                       // [n, nsplit, H, Dvp + 2] partial sums, their maximum and their total, for nsplit > 1
    const int* pos;
    const int* req;
    const int* page_table;
    const void* k_pages;               // [pages, G, 64, Dp]
    const void* v_pages;               // [pages, G, 64, Dvp]
    const float* sink;                 // [H] or null
    const void* gate;                  // [n][H] of pitch gate_ld, in the type of q, or null
    long long gate_ld;
    int pos_stride, req_stride, pt_stride, n_pages;
    int n, H, G, Dp, Dv, Dvp, window, keep, nsplit, kcap;
    float scale_log2;                  // scale times log2(e)
    int* status;
};

// What a query at `pos` sees as one list: element e is position e while e < kept, else lo + e - kept.
struct Seen { int lo, kept, count; };
__device__ __forceinline__ Seen seen_by(int pos, int window, int keep) {
    Seen s;
    s.lo = max(0, pos - window + 1);
    s.kept = min(keep, s.lo);
    s.count = max(0, s.kept + pos - s.lo + 1);
    return s;
}

}  // namespace ptb
