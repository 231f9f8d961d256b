// A short causal convolution over time on each channel:
//   u_t[c] = a(r * y_t[c] + b[c] + sum_{j < taps} w[c, j] * y_(t - taps + 1 + j)[c]),   y before the sequence's start = 0,
// with r = 1 (the convolution is added to its own input) or 0, an optional bias b and a = nothing or SiLU.
// The taps - 1 inputs before a step's first token are the request's state ([slots, taps - 1, channels], fp32,
// oldest first; zero when the request is admitted), so a sequence may be cut into steps anywhere.
//
// Two launches.  `apply` is parallel over (token, channel) and only READS the state: a token whose tap reaches
// back before the step takes it from the state, otherwise from the step's own rows.  `advance` then moves the
// state on, one thread per (request, channel) walking the taps - 1 places in ascending order (with fewer new
// tokens than places, a place takes the value of a later place, which that thread has not overwritten yet).
// In one launch, a block that advanced the state could overtake a block that still reads it.  A step in which every
// request brings ONE token needs neither: one thread per (request, channel) reads the state, forms the output and
// shifts the state by one place, in one launch.
#include "common.cuh"

namespace {

template <typename T>
__global__ void __launch_bounds__(256) short_conv_apply_kernel(
    const T* y, int ldy, T* __restrict__ out, int ldo, const float* __restrict__ w, const float* state,
    const int* __restrict__ token_seq, const int* __restrict__ positions, const int* __restrict__ seq_start_pos,
    const int* __restrict__ seq_state_slot, int channels, int taps, const float* __restrict__ bias, int residual, int act) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int seq = token_seq[t];
    const int pos = positions[t], start = seq_start_pos[seq];
    const int n = taps - 1;
    const float* st = state + (size_t)seq_state_slot[seq] * n * channels;
    const float own = to_float(y[(size_t)t * ldy + c]);
    float acc = (residual ? own : 0.0f) + (bias ? bias[c] : 0.0f);
    const float* wc = w + (size_t)c * taps;
    for (int j = 0; j < taps; ++j) {
        const int back = taps - 1 - j;
        const int p = pos - back;
        float v;
        if (back == 0)
            v = own;
        else if (p < 0)
            v = 0.0f;
        else if (p >= start)
            v = to_float(y[(size_t)(t - back) * ldy + c]);
        else
            v = st[(size_t)(p - start + n) * channels + c];
        acc = fmaf(wc[j], v, acc);
    }
    if (act) acc = acc / (1.0f + expf(-acc));
    out[(size_t)t * ldo + c] = from_float<T>(acc);
}

// `apply` for steps of many tokens: a thread takes two neighbouring channels and SC_RUN tokens in a row, holds the TAPS - 1
// inputs before the next token in registers and reads every row once.  The sums are formed in the same order.
constexpr int SC_RUN = 16;
__device__ __forceinline__ float2 sc_load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 sc_load2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void sc_store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void sc_store2(bf16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

template <typename T, int TAPS>
__global__ void __launch_bounds__(128) short_conv_runs_kernel(
    const T* y, int ldy, T* __restrict__ out, int ldo, const float* __restrict__ w, const float* state,
    const int* __restrict__ token_seq, const int* __restrict__ positions, const int* __restrict__ seq_start_pos,
    const int* __restrict__ seq_state_slot, int tokens, int channels, const float* __restrict__ bias, int residual, int act) {
    constexpr int N = TAPS - 1;
    pdl_wait();
    pdl_launch_dependents();
    const int c = 2 * (blockIdx.y * blockDim.x + threadIdx.x);
    if (c >= channels) return;
    const int t0 = blockIdx.x * SC_RUN, t1 = min(tokens, t0 + SC_RUN);
    float w0[TAPS], w1[TAPS];
#pragma unroll
    for (int j = 0; j < TAPS; ++j) w0[j] = w[(size_t)c * TAPS + j], w1[j] = w[(size_t)(c + 1) * TAPS + j];
    const float2 b = bias ? sc_load2(bias + c) : make_float2(0.0f, 0.0f);
    float2 own[SC_RUN];  // all rows of the run are requested before the first is used
#pragma unroll
    for (int i = 0; i < SC_RUN; ++i)
        if (t0 + i < t1) own[i] = sc_load2(y + (size_t)(t0 + i) * ldy + c);
    float2 past[N > 0 ? N : 1];  // the inputs N, N - 1, .. 1 positions before the token
    int seq = -1;
#pragma unroll
    for (int i = 0; i < SC_RUN; ++i) {
        const int t = t0 + i;
        if (t >= t1) break;
        if (token_seq[t] != seq) {  // the run's or a request's first token: rows of the step before it, else the state
            seq = token_seq[t];
            const int pos = positions[t], start = seq_start_pos[seq];
            const float* st = state + (size_t)seq_state_slot[seq] * N * channels + c;
#pragma unroll
            for (int j = 0; j < N; ++j) {
                const int back = N - j, p = pos - back;
                past[j] = make_float2(0.0f, 0.0f);
                if (p >= start)
                    past[j] = sc_load2(y + (size_t)(t - back) * ldy + c);
                else if (p >= 0)
                    past[j] = sc_load2(st + (size_t)(p - start + N) * channels);
            }
        }
        float a0 = (residual ? own[i].x : 0.0f) + b.x, a1 = (residual ? own[i].y : 0.0f) + b.y;
#pragma unroll
        for (int j = 0; j < N; ++j) a0 = fmaf(w0[j], past[j].x, a0), a1 = fmaf(w1[j], past[j].y, a1);
        a0 = fmaf(w0[N], own[i].x, a0), a1 = fmaf(w1[N], own[i].y, a1);
        if (act) a0 = a0 / (1.0f + expf(-a0)), a1 = a1 / (1.0f + expf(-a1));
        sc_store2(out + (size_t)t * ldo + c, a0, a1);
#pragma unroll
        for (int j = 0; j + 1 < N; ++j) past[j] = past[j + 1];
        if (N > 0) past[N - 1] = own[i];
    }
}

template <typename T>
__global__ void __launch_bounds__(256) short_conv_advance_kernel(const T* y, int ldy, float* state,
                                                                 const int* __restrict__ seq_q_start,
                                                                 const int* __restrict__ seq_state_slot, int channels,
                                                                 int taps) {
    pdl_wait();
    pdl_launch_dependents();
    const int seq = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int n = taps - 1;
    const int row0 = seq_q_start[seq], len = seq_q_start[seq + 1] - row0;
    if (len <= 0) return;
    float* st = state + (size_t)seq_state_slot[seq] * n * channels;
    for (int k = 0; k < n; ++k) {
        const int idx = k + len;  // place in [the old state | the step's rows], of which the last n are kept
        st[(size_t)k * channels + c] = idx < n ? st[(size_t)idx * channels + c] : to_float(y[(size_t)(row0 + idx - n) * ldy + c]);
    }
}

template <typename T>
__global__ void __launch_bounds__(256) short_conv_single_kernel(const T* y, int ldy, T* __restrict__ out, int ldo,
                                                                const float* __restrict__ w, float* state,
                                                                const int* __restrict__ positions,
                                                                const int* __restrict__ seq_state_slot, int channels,
                                                                int taps, const float* __restrict__ bias, int residual,
                                                                int act) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;  // the request's only row of the step
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= channels) return;
    const int n = taps - 1;
    const int pos = positions[t];
    float* st = state + (size_t)seq_state_slot[t] * n * channels + c;
    const float* wc = w + (size_t)c * taps;
    const float own = to_float(y[(size_t)t * ldy + c]);
    float acc = (residual ? own : 0.0f) + (bias ? bias[c] : 0.0f);
    for (int j = 0; j < n; ++j) {  // place j of the state is the input n - j positions back
        const float v = st[(size_t)j * channels];
        if (j > 0) st[(size_t)(j - 1) * channels] = v;
        acc = fmaf(wc[j], pos - (n - j) >= 0 ? v : 0.0f, acc);
    }
    acc = fmaf(wc[n], own, acc);
    if (n > 0) st[(size_t)(n - 1) * channels] = own;
    if (act) acc = acc / (1.0f + expf(-acc));
    out[(size_t)t * ldo + c] = from_float<T>(acc);
}

}  // namespace

// y, out: [tokens, channels] rows ldy / ldo apart (out must not be y); w: fp32 [channels, taps];
// state: fp32 [slots, taps - 1, channels] (may be null when taps == 1); bias: fp32 [channels] or null; residual: the
// input is added to the convolution; act: 0 nothing, 1 SiLU of the sum.
FERRIS_API int ferris_short_conv(const void* y, int ldy, void* out, int ldo, int dtype, const float* w, float* state,
                                 const int* token_seq, const int* positions, const int* seq_q_start,
                                 const int* seq_start_pos, const int* seq_state_slot, int tokens, int seqs, int channels,
                                 int taps, int advance, int single_tokens, const float* bias, int residual, int act,
                                 void* stream) {
    if (tokens <= 0 || seqs <= 0) return FERRIS_OK;
    if (channels <= 0 || taps <= 0) FERRIS_REFUSE("short conv: channels=%d taps=%d", channels, taps);
    if (taps > 1 && !state) FERRIS_REFUSE("short conv: %d taps need a state", taps);
    if (y == out) FERRIS_REFUSE("short conv: input and output must differ");
    cudaStream_t s = (cudaStream_t)stream;
    const int threads = channels >= 256 ? 256 : ((channels + 31) / 32) * 32;
    const int tiles = (channels + threads - 1) / threads;
    if (tiles > 65535) FERRIS_REFUSE("short conv: %d channels are more than one launch takes", channels);
    const dim3 block(threads), grid_a(tokens, tiles), grid_b(seqs, tiles);
    if (single_tokens && advance && tokens == seqs && dtype == FERRIS_F32) {
        ferris_launch(short_conv_single_kernel<float>, grid_a, block, 0, s, (const float*)y, ldy, (float*)out, ldo, w, state,
                      positions, seq_state_slot, channels, taps, bias, residual, act);
        FERRIS_LAUNCH_CHECK();
    }
    if (single_tokens && advance && tokens == seqs && dtype == FERRIS_BF16) {
        ferris_launch(short_conv_single_kernel<bf16>, grid_a, block, 0, s, (const bf16*)y, ldy, (bf16*)out, ldo, w, state,
                      positions, seq_state_slot, channels, taps, bias, residual, act);
        FERRIS_LAUNCH_CHECK();
    }
    const size_t pair = dtype == FERRIS_F32 ? 8 : 4;  // bytes of two channels
    if ((dtype == FERRIS_F32 || dtype == FERRIS_BF16) && tokens >= 2 * SC_RUN && taps >= 2 && taps <= 4 && !((channels | ldy | ldo) & 1) &&
        (uintptr_t)y % pair == 0 && (uintptr_t)out % pair == 0 && (((uintptr_t)state | (uintptr_t)bias) & 7) == 0) {
        const dim3 grid((tokens + SC_RUN - 1) / SC_RUN, (channels / 2 + 127) / 128);
#define FERRIS_SC_RUNS(T, TAPS)                                                                                            \
    ferris_launch(short_conv_runs_kernel<T, TAPS>, grid, dim3(128), 0, s, (const T*)y, ldy, (T*)out, ldo, w, (const float*)state, \
                  token_seq, positions, seq_start_pos, seq_state_slot, tokens, channels, bias, residual, act)
#define FERRIS_SC_TAPS(T)                                                                                                  \
    do {                                                                                                                   \
        if (taps == 2) FERRIS_SC_RUNS(T, 2); else if (taps == 3) FERRIS_SC_RUNS(T, 3); else FERRIS_SC_RUNS(T, 4);            \
        if (advance)                                                                                                       \
            ferris_launch(short_conv_advance_kernel<T>, grid_b, block, 0, s, (const T*)y, ldy, state, seq_q_start,          \
                          seq_state_slot, channels, taps);                                                                 \
    } while (0)
        if (dtype == FERRIS_F32) FERRIS_SC_TAPS(float); else FERRIS_SC_TAPS(bf16);
#undef FERRIS_SC_TAPS
#undef FERRIS_SC_RUNS
        FERRIS_LAUNCH_CHECK();
    }
    if (dtype == FERRIS_F32) {
        ferris_launch(short_conv_apply_kernel<float>, grid_a, block, 0, s, (const float*)y, ldy, (float*)out, ldo, w,
                      (const float*)state, token_seq, positions, seq_start_pos, seq_state_slot, channels, taps, bias, residual, act);
        if (advance && taps > 1)
            ferris_launch(short_conv_advance_kernel<float>, grid_b, block, 0, s, (const float*)y, ldy, state, seq_q_start,
                          seq_state_slot, channels, taps);
    } else if (dtype == FERRIS_BF16) {
        ferris_launch(short_conv_apply_kernel<bf16>, grid_a, block, 0, s, (const bf16*)y, ldy, (bf16*)out, ldo, w,
                      (const float*)state, token_seq, positions, seq_start_pos, seq_state_slot, channels, taps, bias, residual, act);
        if (advance && taps > 1)
            ferris_launch(short_conv_advance_kernel<bf16>, grid_b, block, 0, s, (const bf16*)y, ldy, state, seq_q_start,
                          seq_state_slot, channels, taps);
    } else
        FERRIS_REFUSE("short conv: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}
