// What the forms of the general attention share (attention_simt.cu on CUDA cores in either precision, attention_rows.cu on
// tensor cores in bf16): what enters a score besides the product, which keys a token sees.
#pragma once

#include <math.h>

#include "common.cuh"

namespace {

// What else enters a score and the softmax, per query head (any pointer may be null):
//   slopes:        s_j += slopes[h] * (j - P), a penalty linear in the distance;
//   log_r1, log_r2: s_j -= log_r1[h] * ln(1 + log_r2[h] * (P - j)), a penalty that grows with the distance's logarithm;
//   sink:          the softmax's denominator also holds exp(sink[h]): a weight that belongs to no key and no value;
//   softcap:       the scaled product becomes softcap tanh(product / softcap) ahead of any penalty (0: it stays);
//   gate:          a row of the heads' gates per token (rows ldgate apart, in the queries' type): head h's output is
//                  multiplied by sigmoid(gate[t, h]) where it is stored.
// v_stride: elements between the value rows of consecutive cache rows (0: dv).  With the key cache given as the
// value cache too and v_stride = d, a value is the first dv elements of its key (keys that carry their value).
struct ScoreTerms {
    const float* slopes;
    const float* log_r1;
    const float* log_r2;
    const float* sink;
    int v_stride;
    float softcap;
    const void* gate;
    int ldgate;
};
// Keys that a token sees beside its window, as rows 0, 1, .. ahead of it: k [pages, nkv, page_size, d] and v [.., dv], rows
// addressed by tables [requests, max_blocks] as tokens are by the step's block tables.  Either (every > 0) one row for every
// run of `every` positions that lies wholly before the window, in pages of their own, or (keep > 0) the sequence's first
// `keep` tokens where the window has passed them, in the tokens' own pages.  Kernels with POOL walk the keys by one index
// n: n < ahead_rows(first position of the window) is such a row, the others are the tokens from the window's first position on.
struct PooledKeys {
    const void* k;
    const void* v;
    const int* tables;
    int max_blocks, every, keep;
};
__device__ __forceinline__ int ahead_rows(const PooledKeys& pk, int lo) {
    return pk.every > 0 ? lo / pk.every : (pk.keep < lo ? pk.keep : lo);
}
struct HeadTerms {
    int kind;  // 0: nothing, 1: slope, 2: logarithm
    float a, b;
    float cap;
};
__device__ __forceinline__ HeadTerms head_terms(const ScoreTerms& st, int h) {
    HeadTerms t = {0, 0.0f, 0.0f, st.softcap};
    if (st.slopes) t.kind = 1, t.a = st.slopes[h];
    if (st.log_r1) t.kind = 2, t.a = st.log_r1[h], t.b = st.log_r2[h];
    return t;
}
// the score of the key at j for the query at P, from the scaled product
__device__ __forceinline__ float with_terms(float s, const HeadTerms& t, int j, int P) {
    if (t.cap > 0.0f) s = t.cap * tanhf(s / t.cap);
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

// what the output of head h at token t is multiplied by
template <typename T>
__device__ __forceinline__ float head_gate(const ScoreTerms& st, int t, int h) {
    if (!st.gate) return 1.0f;
    return 1.0f / (1.0f + expf(-to_float(reinterpret_cast<const T*>(st.gate)[(size_t)t * st.ldgate + h])));
}

// Whether the arguments for pooled keys make sense (all null / 0: there are none).
int check_pooled(const PooledKeys& pk, int window, const ScoreTerms& st) {
    if (st.softcap < 0.0f) FERRIS_REFUSE("attention: a soft cap of %g", (double)st.softcap);
    if (pk.keep < 0 || (pk.keep > 0 && pk.every > 0)) FERRIS_REFUSE("attention: %d kept tokens beside pooled keys of %d", pk.keep, pk.every);
    if (pk.keep > 0) {
        if (window <= 0) FERRIS_REFUSE("attention: kept tokens stand before a window");
        return FERRIS_OK;
    }
    if (pk.every == 0 && !pk.k && !pk.v && !pk.tables) return FERRIS_OK;
    if (pk.every <= 0 || !pk.k || !pk.v || !pk.tables || pk.max_blocks <= 0)
        FERRIS_REFUSE("attention: pooled keys of %d positions want rows and block tables", pk.every);
    if (window <= 0) FERRIS_REFUSE("attention: pooled keys stand before a window");
    if (st.slopes || st.log_r1 || st.v_stride) FERRIS_REFUSE("attention: pooled keys go with no distance penalty and no values in keys");
    return FERRIS_OK;
}

// The keys beside the window that a launcher was given: pooled rows, kept tokens of the step's own pages, or none.
PooledKeys keys_beside(const void* pool_k, const void* pool_v, const int* pool_tables, int pool_max_blocks, int pool_every,
                       int keep, const void* k_cache, const void* v_cache, const int* block_tables, int max_blocks) {
    if (keep > 0 && pool_every == 0) return {k_cache, v_cache, block_tables, max_blocks, 0, keep};
    return {pool_k, pool_v, pool_tables, pool_max_blocks, pool_every, keep};
}

}  // namespace
