// Options of the attention kernels that differ between designs: which positions a query sees, how its scores are transformed,
// what joins the denominator and how the output is gated.  One struct, passed by pointer through the C entry points (null: plain
// causal attention) and by value into the kernels.
#pragma once

#include "ps_common.cuh"

namespace ps {

struct AttnOptions {
    int chunk;                   // > 0: position i sees only its own block of `chunk` positions (counted from position 0)
    int window;                  // > 0: position i sees only positions j with i - j < window
    float temp_coef, temp_every; // scores of a query at position p are multiplied by 1 + coef ln(floor((p + 1) / every) + 1)
    const float* bias;           // [Hq, bias_len] or null: added to the score of a key at distance i - j (last entry: and beyond)
    int bias_len;
    int gate_per_head;           // the sigmoid gate is one number per head instead of one per element
    const float* sink;           // [Hq] or null: exp(sink[h]) joins head h's denominator
    int keep_first;              // > 0: the first `keep_first` positions of the sequence are seen besides the window or block
};

// First position of the run up to `pos` itself that a query at `pos` sees (kept first positions lie before it).
__device__ __forceinline__ int attn_first(const AttnOptions& o, int pos) {
    int lo = o.chunk > 0 ? pos / o.chunk * o.chunk : 0;
    if (o.window > 0) lo = max(lo, pos - o.window + 1);
    return lo;
}
// Whether a query whose run begins at `lo` sees position `tok` (not later than the query).
__device__ __forceinline__ bool attn_sees(const AttnOptions& o, int lo, int tok) { return tok >= lo || tok < o.keep_first; }
__device__ __forceinline__ float attn_temperature(const AttnOptions& o, int pos) {
    if (o.temp_coef == 0.f) return 1.f;
    return 1.f + o.temp_coef * logf((float)(floor((double)(pos + 1) / (double)o.temp_every) + 1.0));
}
// Bias of query head `h` for a key `dist` >= 0 positions back.
__device__ __forceinline__ float attn_bias(const AttnOptions& o, int h, int dist) {
    return o.bias == nullptr ? 0.f : __ldg(o.bias + (size_t)h * o.bias_len + min(dist, o.bias_len - 1));
}

inline AttnOptions attn_options(const void* p) {
    if (p != nullptr) return *static_cast<const AttnOptions*>(p);
    AttnOptions o = {};
    o.temp_every = 1.f;
    return o;
}
inline bool attn_options_ok(const AttnOptions& o) {
    return o.chunk >= 0 && o.window >= 0 && o.keep_first >= 0 && (o.bias == nullptr || o.bias_len > 0) && o.temp_every > 0.f;
}
// Scores need more than the scale before their maximum is taken.
inline bool attn_transforms_scores(const AttnOptions& o) { return o.bias != nullptr || o.temp_coef != 0.f; }

}  // namespace ps
