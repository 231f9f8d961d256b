// What the forms of the general attention share (attention_simt.cu on CUDA cores in either precision, attention_rows.cu on
// tensor cores in bf16): what enters a score besides the product, which keys a token sees, the merge of shares.
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

// out = sum_s o_s e^(m_s - M) / sum_s z_s e^(m_s - M) over the shares of the keys that the kernel above left in `partial`
// ([tokens, heads, splits, 2 + dv]: maximum, sum, weighted values).  A block per (token, head).
template <typename T>
__global__ void __launch_bounds__(128) attention_merge_shares_kernel(const float* partial, T* __restrict__ out, int ldo,
                                                                     int nh, int dv, int splits, const ScoreTerms st) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x, h = blockIdx.y;
    const int stride = dv + 2;
    const float* base = partial + ((size_t)t * nh + h) * splits * stride;
    float mm = -INFINITY;
    for (int s2 = 0; s2 < splits; ++s2) mm = fmaxf(mm, base[(size_t)s2 * stride]);
    float zz = 0.0f;
    for (int s2 = 0; s2 < splits; ++s2) {
        const float ms = base[(size_t)s2 * stride];
        zz += ms == -INFINITY ? 0.0f : base[(size_t)s2 * stride + 1] * expf(ms - mm);
    }
    zz += sink_share(st, h, mm);
    const float inv = 1.0f / zz;
    for (int i = threadIdx.x; i < dv; i += blockDim.x) {
        float o = 0.0f;
        for (int s2 = 0; s2 < splits; ++s2) {
            const float ms = base[(size_t)s2 * stride];
            if (ms != -INFINITY) o += base[(size_t)s2 * stride + 2 + i] * expf(ms - mm);
        }
        out[(size_t)t * ldo + (size_t)h * dv + i] = from_float<T>(o * inv);
    }
}

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
