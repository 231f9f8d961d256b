// What the forms of the general attention share (attention_simt.cu on CUDA cores in either precision, attention_rows.cu on
// tensor cores in bf16): what enters a score besides the product, which keys a token sees.
#pragma once

#include <math.h>

#include "common.cuh"

namespace {

// What else enters a score and the softmax, per query head (any pointer may be null):
//   slopes:        s_j += slopes[h] * (j - P), a penalty linear in the distance;
//   log_r1, log_r2: s_j -= log_r1[h] * ln(1 + log_r2[h] * (P - j)), a penalty that grows with the distance's logarithm;
//   sink:          the softmax's denominator also holds exp(sink[h]): a weight that belongs to no key and no value.
// v_stride: elements between the value rows of consecutive cache rows (0: dv).  With the key cache given as the
// value cache too and v_stride = d, a value is the first dv elements of its key (keys that carry their value).
struct ScoreTerms {
    const float* slopes;
    const float* log_r1;
    const float* log_r2;
    const float* sink;
    int v_stride;
};
// Keys that stand for runs of positions before the window: k [pages, nkv, page_size, d] and v [.., dv], rows addressed by
// tables [requests, max_blocks] as tokens are by the step's block tables.  Kernels with POOL walk the keys by one index
// n: n < pooled is the run n, the others are the tokens from the window's first position on.
struct PooledKeys {
    const void* k;
    const void* v;
    const int* tables;
    int max_blocks, every;
};
struct HeadTerms {
    int kind;  // 0: nothing, 1: slope, 2: logarithm
    float a, b;
};
__device__ __forceinline__ HeadTerms head_terms(const ScoreTerms& st, int h) {
    HeadTerms t = {0, 0.0f, 0.0f};
    if (st.slopes) t.kind = 1, t.a = st.slopes[h];
    if (st.log_r1) t.kind = 2, t.a = st.log_r1[h], t.b = st.log_r2[h];
    return t;
}
// the score of the key at j for the query at P, from the scaled product
__device__ __forceinline__ float with_terms(float s, const HeadTerms& t, int j, int P) {
    if (t.kind == 1) return fmaf(t.a, (float)(j - P), s);
    if (t.kind == 2) return s - t.a * log1pf(t.b * (float)(P - j));
    return s;
}
// The first key that the query at position P sees.  window > 0: the last `window` keys, itself included; window < 0:
// the keys of its own chunk, positions being counted off in chunks of -window from 0; 0: every key.
__device__ __forceinline__ int first_key(int P, int window) {
    if (window > 0) return P - window + 1 > 0 ? P - window + 1 : 0;
    if (window < 0) return P - P % (-window);
    return 0;
}
// the sink's share of the denominator, relative to the maximum mm of the keys' scores
__device__ __forceinline__ float sink_share(const ScoreTerms& st, int h, float mm) { return st.sink ? expf(st.sink[h] - mm) : 0.0f; }

// Whether the arguments for pooled keys make sense (all null / 0: there are none).
int check_pooled(const PooledKeys& pk, int window, const ScoreTerms& st) {
    if (pk.every == 0 && !pk.k && !pk.v && !pk.tables) return FERRIS_OK;
    if (pk.every <= 0 || !pk.k || !pk.v || !pk.tables || pk.max_blocks <= 0)
        FERRIS_REFUSE("attention: pooled keys of %d positions want rows and block tables", pk.every);
    if (window <= 0) FERRIS_REFUSE("attention: pooled keys stand before a window");
    if (st.slopes || st.log_r1 || st.v_stride) FERRIS_REFUSE("attention: pooled keys go with no distance penalty and no values in keys");
    return FERRIS_OK;
}

}  // namespace
