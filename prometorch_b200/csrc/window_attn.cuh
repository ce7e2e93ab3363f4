// Softmax attention over the paged cache.  The query at position p sees the keys from `low(p)` to p and the first `keep` tokens of its
// sequence; low is p - window + 1 (a sliding window) or, chunked, the first position of p's chunk of `window` positions.  A sink adds
// exp(sink_h) to a head's denominator; a gate scales the head's output by its sigmoid.
// A distance bias adds rel[h][min(p - j, rel_n - 1)] to the scaled score of key j.
// Two maps: q and k of a head are [map 1, map 2], each an attention of its own over the same values, and the output is
// d / sqrt(mean(d^2) + mix_eps) * mix_gain with d = a1 - mix a2.
#pragma once
#include "common.cuh"
#include "ptb200_types.h"

namespace ptb {

constexpr int WA_PAGE = 64;
constexpr int WA_KEYS = 128;           // most keys of one CTA of the row kernels
constexpr int WA_HEADS = 32;           // most query heads of one CTA of the row kernels (64 with two maps)
constexpr float WA_LOG2E = 1.4426950408889634f;

// First position that the query at `pos` sees besides the kept ones.
__device__ __forceinline__ int low_of(int pos, int window, int chunked) { return chunked ? pos - pos % window : max(0, pos - window + 1); }

// What a query at `pos` sees as one list: element e is position e while e < kept, else lo + e - kept.
struct Seen { int lo, kept, count; };
__device__ __forceinline__ Seen seen_by(int pos, int window, int keep, int chunked) {
    Seen s;
    s.lo = low_of(max(pos, 0), window, chunked);
    s.kept = min(keep, s.lo);
    s.count = max(0, s.kept + pos - s.lo + 1);
    return s;
}

}  // namespace ptb
