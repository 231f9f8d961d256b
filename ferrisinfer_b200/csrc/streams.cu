// What stands around the mixers of layers that keep several residual streams, shift their input by a token, run two
// mixers side by side, or attend over a shared latent instead of per-head keys and values.
//
// Residual streams (hyper-connections): instead of one residual row a token has S of them, [tokens, S, width] fp32.
// A sublayer reads u = sum_s in[s] x_s through its norm, and its result y goes back as
//   x_r <- sum_s mix[s, r] x_s + out[r] y      for all r at once, from the old streams.
// `streams_step` does the write of one sublayer and the read (with the RMS norm) of the next in one pass over the
// token's streams; either half may be left out.
#include <math.h>

#include "common.cuh"
#include "sm100.cuh"

namespace {

constexpr int MAX_STREAMS = 8;

struct StreamWeights {
    float mix[MAX_STREAMS * MAX_STREAMS];  // [from, to]
    float out[MAX_STREAMS];
    float in[MAX_STREAMS];
};

__global__ void __launch_bounds__(256) streams_expand_kernel(const float* h, float* __restrict__ xs, int streams, int width) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float v = h[(size_t)t * width + c];
        for (int s = 0; s < streams; ++s) xs[((size_t)t * streams + s) * width + c] = v;
    }
}

__global__ void __launch_bounds__(256) streams_sum_kernel(const float* xs, float* __restrict__ h, int streams, int width) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float v = 0.0f;
        for (int s = 0; s < streams; ++s) v += xs[((size_t)t * streams + s) * width + c];
        h[(size_t)t * width + c] = v;
    }
}

// write (y not null): the streams take the sublayer's result; read (norm_w not null): out = rmsnorm(sum_s in[s] x_s) * norm_w.
// mix, out_w, in_w lie in device memory (learned tensors), fp32.
template <typename T>
__global__ void __launch_bounds__(512) streams_step_kernel(float* xs, const float* y, const float* __restrict__ mix,
                                                           const float* __restrict__ out_w, const float* __restrict__ in_w,
                                                           const float* __restrict__ norm_w, float eps, T* __restrict__ out,
                                                           int streams, int width, const float* __restrict__ shift,
                                                           float* shift_state, const int* __restrict__ positions,
                                                           const int* __restrict__ seq_state_slot) {
    extern __shared__ float u_row[];  // [width], the read's sum (only with a read)
    __shared__ float scratch[33];
    __shared__ StreamWeights sw;
    const bool writes = y != nullptr, reads = norm_w != nullptr;
    // the learned numbers are weights: they may be read before the launch before this one has ended
    if (threadIdx.x < streams * streams && writes) sw.mix[threadIdx.x] = mix[threadIdx.x];
    if (threadIdx.x < streams) {
        if (writes) sw.out[threadIdx.x] = out_w[threadIdx.x];
        if (reads) sw.in[threadIdx.x] = in_w[threadIdx.x];
    }
    __syncthreads();
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    float* row = xs + (size_t)t * streams * width;
    float ss = 0.0f;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float x[MAX_STREAMS];
#pragma unroll
        for (int s = 0; s < MAX_STREAMS; ++s) x[s] = s < streams ? row[(size_t)s * width + c] : 0.0f;
        if (writes) {
            const float yy = y[(size_t)t * width + c];
            float nx[MAX_STREAMS];
#pragma unroll
            for (int r = 0; r < MAX_STREAMS; ++r) {
                float a = 0.0f;
                if (r < streams) {
#pragma unroll
                    for (int s = 0; s < MAX_STREAMS; ++s)
                        if (s < streams) a = fmaf(sw.mix[s * streams + r], x[s], a);
                    a = fmaf(sw.out[r], yy, a);
                    row[(size_t)r * width + c] = a;
                }
                nx[r] = a;
            }
#pragma unroll
            for (int r = 0; r < MAX_STREAMS; ++r) x[r] = nx[r];
        }
        if (reads) {
            float u = 0.0f;
#pragma unroll
            for (int s = 0; s < MAX_STREAMS; ++s)
                if (s < streams) u = fmaf(sw.in[s], x[s], u);
            u_row[c] = u;
            ss = fmaf(u, u, ss);
        }
    }
    if (!reads) return;
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)width + eps);
    if (!shift) {
        for (int c = threadIdx.x; c < width; c += blockDim.x) out[(size_t)t * width + c] = from_float<T>((u_row[c] * inv) * norm_w[c]);
        return;
    }
    // A step of single tokens (row t is request t's only token): the token shift of the normed row right here, from and
    // to the request's state, on the row as it is rounded for the mixer (what the kernels of its own do as well).
    const int pos = positions[t];
    float* st = shift_state + (size_t)seq_state_slot[t] * width;
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        const float own = to_float(from_float<T>((u_row[c] * inv) * norm_w[c]));
        const float prev = pos == 0 ? 0.0f : st[c];
        st[c] = own;
        out[(size_t)t * width + c] = from_float<T>(fmaf(prev - own, shift[c], own));
    }
}

// ---------------------------------------------------------------------------------------------
// Token shift: a mixer's input row x_t becomes x_t + (x_(t-1) - x_t) * shift, with x_(t-1) the row of the token before
// as it was BEFORE its own shift (zeros for a sequence's first token).  The last unshifted row of a request is its
// state ([slots, width] fp32).  `apply` only reads the state and `advance` then writes it (a block that advanced it
// could otherwise overtake one that still reads it); a step of single tokens does both in one launch.
// ---------------------------------------------------------------------------------------------
template <typename T>
__global__ void __launch_bounds__(256) token_shift_apply_kernel(const T* x, T* __restrict__ out, const float* __restrict__ shift,
                                                                float* state, const int* __restrict__ token_seq,
                                                                const int* __restrict__ positions,
                                                                const int* __restrict__ seq_start_pos,
                                                                const int* __restrict__ seq_state_slot, int width, int single) {
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= width) return;
    const int seq = token_seq[t];
    const int pos = positions[t];
    float* st = state + (size_t)seq_state_slot[seq] * width + c;
    const float own = to_float(x[(size_t)t * width + c]);
    float prev;
    if (pos == 0)
        prev = 0.0f;
    else if (pos == seq_start_pos[seq])
        prev = *st;
    else
        prev = to_float(x[(size_t)(t - 1) * width + c]);
    out[(size_t)t * width + c] = from_float<T>(fmaf(prev - own, shift[c], own));
    if (single) *st = own;
}

template <typename T>
__global__ void __launch_bounds__(256) token_shift_advance_kernel(const T* x, float* state, const int* __restrict__ seq_q_start,
                                                                  const int* __restrict__ seq_state_slot, int width) {
    pdl_wait();
    pdl_launch_dependents();
    const int seq = blockIdx.x;
    const int c = blockIdx.y * blockDim.x + threadIdx.x;
    if (c >= width) return;
    const int last = seq_q_start[seq + 1] - 1;
    if (last < seq_q_start[seq]) return;
    state[(size_t)seq_state_slot[seq] * width + c] = to_float(x[(size_t)last * width + c]);
}

// ---------------------------------------------------------------------------------------------
// Mixers side by side: h += coef * sum_b rmsnorm(y_b) * w_b over up to four branches' results (fp32 rows).
// ---------------------------------------------------------------------------------------------
struct Branches {
    const float* y[4];
    const float* w[4];
    int n;
};

__global__ void __launch_bounds__(256) branch_norm_sum_kernel(Branches br, float coef, float eps, float* h, int width,
                                                              int accumulate) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    float inv[4];
#pragma unroll
    for (int b = 0; b < 4; ++b) {
        inv[b] = 0.0f;
        if (b < br.n) {
            float ss = 0.0f;
            for (int c = threadIdx.x; c < width; c += blockDim.x) {
                const float v = br.y[b][(size_t)t * width + c];
                ss = fmaf(v, v, ss);
            }
            ss = block_sum(ss, scratch);
            inv[b] = 1.0f / sqrtf(ss / (float)width + eps);
        }
    }
    for (int c = threadIdx.x; c < width; c += blockDim.x) {
        float a = 0.0f;
#pragma unroll
        for (int b = 0; b < 4; ++b)
            if (b < br.n) a += (br.y[b][(size_t)t * width + c] * inv[b]) * br.w[b][c];
        h[(size_t)t * width + c] = accumulate ? fmaf(coef, a, h[(size_t)t * width + c]) : coef * a;
    }
}

// ---------------------------------------------------------------------------------------------
// Attention over a shared latent.  A token's projection row holds [rank latent | rot rotated key] dimensions; its query rows
// hold, per head, [dim plain | rot rotated] dimensions (in the same projection row, or, where queries go through a latent of
// their own, in the rows of a later product).  Three pieces of work, any of which may be left out of a launch:
//   keys       the latent is normed (RMS norm with a weight), the key part rotated, [latent | rotated key] written as the
//              token's one cache row;
//   queries    the heads' rotated query parts go into the attention's query rows behind the place of the absorbed plain part:
//              q_att[t, h] = [rank: left for the product of the plain query with the key up-projection | rot: rotated part];
//   q latent   the query latent is normed (RMS norm with a weight of its own) into rows for the next product.
// Rotation: the first `rot_dims` of the part, elements (i, i + rot_dims / 2) or (2i, 2i + 1) together (interleaved), angle =
// position * freq[i] in fp32; with freq_lo (what the 32-bit frequencies lack of their 64-bit values) the angle keeps the digits
// that one 32-bit product rounds away.
// ---------------------------------------------------------------------------------------------
struct LatentArgs {
    const void* q;  // null: no queries
    const void* dkv;  // null: no keys
    const void* cq;  // null: no query latent
    void* cq_out;
    const float* cq_norm;
    const float* norm;
    const float* freq;
    const float* freq_lo;
    const int* positions;
    const int* slots;
    void* cache;
    void* q_att;
    int ldq, lddkv, ldcq, ldcq_out, ldqa, q_rank, rot_dims, interleaved, heads, dim, rot, rank;
    float eps;
};

template <typename T>
__device__ __forceinline__ float rotated(const T* src, int e, int rot_dims, int interleaved, const float* cs, const float* sn) {
    const float v = to_float(src[e]);
    if (e >= rot_dims) return v;
    const int half = rot_dims >> 1;
    const bool first = interleaved ? !(e & 1) : e < half;
    const int f = interleaved ? e >> 1 : (first ? e : e - half);
    const float other = to_float(src[interleaved ? (e ^ 1) : (first ? e + half : e - half)]);
    return first ? v * cs[f] - other * sn[f] : v * cs[f] + other * sn[f];
}

template <typename T>
__device__ __forceinline__ void normed_row(const T* src, T* dst, int n, const float* __restrict__ w, float eps, float* scratch) {
    float ss = 0.0f;
    for (int i = threadIdx.x; i < n; i += blockDim.x) {
        const float v = to_float(src[i]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
    for (int i = threadIdx.x; i < n; i += blockDim.x) dst[i] = from_float<T>((to_float(src[i]) * inv) * w[i]);
}

template <typename T>
__global__ void __launch_bounds__(128) latent_prepare_kernel(const LatentArgs p) {
    __shared__ float scratch[33];
    __shared__ float cs[256], sn[256];  // the token's angles, once for the key part and every head
    pdl_wait();
    pdl_launch_dependents();
    // the pieces of a token side by side: blockIdx.y 0 takes keys and queries, 1 the query latent
    const int t = blockIdx.x;
    if (p.cq && (blockIdx.y == 1 || gridDim.y == 1)) {
        normed_row(reinterpret_cast<const T*>(p.cq) + (size_t)t * p.ldcq, reinterpret_cast<T*>(p.cq_out) + (size_t)t * p.ldcq_out,
                   p.q_rank, p.cq_norm, p.eps, scratch);
        if (gridDim.y > 1) return;
        __syncthreads();
    }
    if (!p.q && !p.dkv) return;
    const float pos = (float)p.positions[t];
    for (int f = threadIdx.x; f < (p.rot_dims >> 1); f += blockDim.x) {
        const float hi = p.freq[f], angle = pos * hi;
        float s, c;
        sincosf(angle, &s, &c);
        if (p.freq_lo) {  // sin(a + e) = sin a + e cos a, cos(a + e) = cos a - e sin a
            const float e = fmaf(pos, hi, -angle) + pos * p.freq_lo[f];
            const float s0 = s;
            s = fmaf(e, c, s), c = fmaf(-e, s0, c);
        }
        cs[f] = c, sn[f] = s;
    }
    __syncthreads();
    if (p.q) {
        const T* row = reinterpret_cast<const T*>(p.q) + (size_t)t * p.ldq;
        T* dst = reinterpret_cast<T*>(p.q_att) + (size_t)t * p.ldqa;
        for (int i = threadIdx.x; i < p.heads * p.rot; i += blockDim.x) {
            const int h = i / p.rot, e = i - h * p.rot;
            const float v = rotated(row + (size_t)h * (p.dim + p.rot) + p.dim, e, p.rot_dims, p.interleaved, cs, sn);
            dst[(size_t)h * (p.rank + p.rot) + p.rank + e] = from_float<T>(v);
        }
    }
    if (!p.dkv) return;
    const T* dkv = reinterpret_cast<const T*>(p.dkv) + (size_t)t * p.lddkv;
    T* dst = reinterpret_cast<T*>(p.cache) + (size_t)p.slots[t] * (p.rank + p.rot);
    for (int e = threadIdx.x; e < p.rot; e += blockDim.x)
        dst[p.rank + e] = from_float<T>(rotated(dkv + p.rank, e, p.rot_dims, p.interleaved, cs, sn));
    normed_row(dkv, dst, p.rank, p.norm, p.eps, scratch);
}

// ---------------------------------------------------------------------------------------------
// A small product per head: out[t, h, n] = (sum_k x[t, h, k] W[h, k, n]) * g, g = 1 or sigmoid(gate[t, h]).
// Eight tokens of a head stand in shared memory (fp32); a thread owns an output column for all eight and a quarter
// of the inputs, and reads each of its weights once, consecutive threads consecutive columns; the four quarters'
// sums are added in order.  fp32 FMAs.
// ---------------------------------------------------------------------------------------------
constexpr int HG_TOKENS = 8, HG_COLS = 64, HG_PARTS = 4, HG_THREADS = HG_COLS * HG_PARTS;

template <typename T>
__global__ void __launch_bounds__(HG_THREADS) head_gemm_kernel(const T* x, int ldx, int hsx, const T* __restrict__ w, T* __restrict__ out,
                                                               int ldo, int hso, const T* gate, int ldg, int tokens, int K,
                                                               int N) {
    extern __shared__ float xs[];  // [HG_TOKENS][K], then the parts' sums [HG_PARTS - 1][HG_TOKENS][HG_COLS]
    pdl_wait();
    pdl_launch_dependents();
    const int t0 = blockIdx.x * HG_TOKENS, h = blockIdx.y;
    const int cl = threadIdx.x % HG_COLS, part = threadIdx.x / HG_COLS;
    const int n = blockIdx.z * HG_COLS + cl;
    const int rows = tokens - t0 < HG_TOKENS ? tokens - t0 : HG_TOKENS;
    for (int i = threadIdx.x; i < HG_TOKENS * K; i += HG_THREADS) {
        const int r = i / K, k = i - r * K;
        xs[i] = r < rows ? to_float(x[(size_t)(t0 + r) * ldx + (size_t)h * hsx + k]) : 0.0f;
    }
    __syncthreads();
    // the inputs are cut into four runs, a quarter of the block each: four times as many weights are on their way
    float acc[HG_TOKENS];
#pragma unroll
    for (int r = 0; r < HG_TOKENS; ++r) acc[r] = 0.0f;
    const int per = (K + HG_PARTS - 1) / HG_PARTS;
    const int k0 = part * per, k1 = min(K, k0 + per);
    if (n < N) {
        const T* wh = w + (size_t)h * K * N + n;
#pragma unroll 8
        for (int k = k0; k < k1; ++k) {
            const float wv = to_float(wh[(size_t)k * N]);
#pragma unroll
            for (int r = 0; r < HG_TOKENS; ++r) acc[r] = fmaf(xs[r * K + k], wv, acc[r]);
        }
    }
    float* sums = xs + HG_TOKENS * K;
    if (part > 0) {
#pragma unroll
        for (int r = 0; r < HG_TOKENS; ++r) sums[((part - 1) * HG_TOKENS + r) * HG_COLS + cl] = acc[r];
    }
    __syncthreads();
    if (part > 0 || n >= N) return;
#pragma unroll
    for (int r = 0; r < HG_TOKENS; ++r) {
        if (r >= rows) break;
        float v = acc[r];
#pragma unroll
        for (int p = 0; p < HG_PARTS - 1; ++p) v += sums[(p * HG_TOKENS + r) * HG_COLS + cl];  // in the runs' order
        if (gate) v *= 1.0f / (1.0f + expf(-to_float(gate[(size_t)(t0 + r) * ldg + h])));
        out[(size_t)(t0 + r) * ldo + (size_t)h * hso + n] = from_float<T>(v);
    }
}

// The same product for long bf16 steps on the tensor cores: a block takes 64 tokens and 64 output columns of a head and walks
// the inputs 64 at a time through two stages of asynchronous copies; each of its four warps owns 16 tokens.  bf16 operands as
// stored, fp32 sums.
constexpr int HM_TOKENS = 64, HM_COLS = 64, HM_K = 64, HM_THREADS = 128;
constexpr int HM_PITCH = (HM_K + 8) * 2;  // bytes of a row of either tile: eight rows lie in different banks

__device__ __forceinline__ void hm_copy16(uint32_t dst, const void* src, bool there) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(there ? 16 : 0) : "memory");
}

__global__ void __launch_bounds__(HM_THREADS) head_gemm_mma_kernel(const bf16* x, int ldx, int hsx, const bf16* __restrict__ w,
                                                                   bf16* __restrict__ out, int ldo, int hso, const bf16* gate,
                                                                   int ldg, int tokens, int K, int N) {
    __shared__ __align__(16) uint8_t xs[2][HM_TOKENS * HM_PITCH];
    __shared__ __align__(16) uint8_t wt[2][HM_K * HM_PITCH];
    pdl_wait();
    pdl_launch_dependents();
    const int t0 = blockIdx.x * HM_TOKENS, h = blockIdx.y, n0 = blockIdx.z * HM_COLS;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const bf16* wh = w + (size_t)h * K * N;
    auto fetch = [&](int k0, int st) {
        if (k0 < K) {
            const uint32_t xb = smem_u32(xs[st]), wb = smem_u32(wt[st]);
#pragma unroll
            for (int it = 0; it < HM_TOKENS * (HM_K / 8) / HM_THREADS; ++it) {
                const int e = it * HM_THREADS + tid, r = e >> 3, c = (e & 7) * 8;
                const bool in = t0 + r < tokens && k0 + c < K;
                hm_copy16(xb + r * HM_PITCH + c * 2, in ? x + (size_t)(t0 + r) * ldx + (size_t)h * hsx + k0 + c : x, in);
                const bool win = k0 + r < K && n0 + c < N;  // the weights' tile has as many rows (inputs) and pieces
                hm_copy16(wb + r * HM_PITCH + c * 2, win ? wh + (size_t)(k0 + r) * N + n0 + c : wh, win);
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    float acc[HM_COLS / 8][4];
#pragma unroll
    for (int n = 0; n < HM_COLS / 8; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[n][e] = 0.0f;
    fetch(0, 0);
    int st = 0;
    for (int k0 = 0; k0 < K; k0 += HM_K, st ^= 1) {
        fetch(k0 + HM_K, st ^ 1);
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();
        const uint32_t a_at = smem_u32(xs[st]) + (uint32_t)(16 * warp + (lane & 7) + ((lane >> 3) & 1) * 8) * HM_PITCH + (lane >> 4) * 16;
        const uint32_t b_at = smem_u32(wt[st]) + (uint32_t)(((lane >> 3) & 1) * 8 + (lane & 7)) * HM_PITCH + (lane >> 4) * 16;
#pragma unroll
        for (int kk = 0; kk < HM_K / 16; ++kk) {
            uint32_t a[4];
            ldmatrix_x4(a, a_at + kk * 32);
#pragma unroll
            for (int n = 0; n < HM_COLS / 8; n += 2) {
                uint32_t b[4];
                ldmatrix_x4_trans(b, b_at + kk * 16 * HM_PITCH + n * 16);
                mma_bf16_16816(acc[n], a, b[0], b[1]);
                mma_bf16_16816(acc[n + 1], a, b[2], b[3]);
            }
        }
        __syncthreads();  // the stage is read: the copies after next may overwrite it
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int a = 0; a < 2; ++a) {
        const int t = t0 + 16 * warp + (lane >> 2) + 8 * a;
        if (t >= tokens) continue;
        const float g = gate ? 1.0f / (1.0f + expf(-to_float(gate[(size_t)t * ldg + h]))) : 1.0f;
        bf16* row = out + (size_t)t * ldo + (size_t)h * hso;
#pragma unroll
        for (int n = 0; n < HM_COLS / 8; ++n) {
            const int c = n0 + 8 * n + 2 * (lane & 3);
            if (c < N) *reinterpret_cast<uint32_t*>(row + c) = pack_bf16(acc[n][2 * a] * g, acc[n][2 * a + 1] * g);
        }
    }
}
constexpr int HM_MIN_TOKENS = 48;  // shorter steps keep the kernel above: its blocks of eight tokens fill more SMs

}  // namespace

FERRIS_API int ferris_streams_expand(const float* h, float* xs, int tokens, int streams, int width, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (streams <= 0 || width <= 0) FERRIS_REFUSE("streams: %d streams of %d", streams, width);
    ferris_launch(streams_expand_kernel, dim3(tokens), dim3(width >= 1024 ? 256 : 128), 0, (cudaStream_t)stream, h, xs, streams, width);
    FERRIS_LAUNCH_CHECK();
}

FERRIS_API int ferris_streams_sum(const float* xs, float* h, int tokens, int streams, int width, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (streams <= 0 || width <= 0) FERRIS_REFUSE("streams: %d streams of %d", streams, width);
    ferris_launch(streams_sum_kernel, dim3(tokens), dim3(width >= 1024 ? 256 : 128), 0, (cudaStream_t)stream, xs, h, streams, width);
    FERRIS_LAUNCH_CHECK();
}

// xs: fp32 [tokens, streams, width]; y (null: no write): fp32 [tokens, width] with mix [streams, streams] and out_w
// [streams]; norm_w (null: no read): fp32 [width] with in_w [streams], out: [tokens, width] of `dtype`.  shift (null: none;
// only where every request brings one token, row t being request t's): fp32 [width]; the read's rows are shifted towards
// shift_state[seq_state_slot[t]] (fp32 [slots, width]; zeros at position 0), which takes the unshifted row.
FERRIS_API int ferris_streams_step(float* xs, const float* y, const float* mix, const float* out_w, const float* in_w,
                                   const float* norm_w, float eps, void* out, int dtype, int tokens, int streams, int width,
                                   const float* shift, float* shift_state, const int* positions, const int* seq_state_slot,
                                   void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (streams <= 0 || streams > MAX_STREAMS || width <= 0) FERRIS_REFUSE("streams: %d streams (at most %d) of %d", streams, MAX_STREAMS, width);
    if (y && (!mix || !out_w)) FERRIS_REFUSE("streams: a write needs its mixing matrix and output weights");
    if (norm_w && (!in_w || !out)) FERRIS_REFUSE("streams: a read needs its input weights and an output");
    if (!y && !norm_w) return FERRIS_OK;
    if (shift && (!norm_w || !shift_state || !positions || !seq_state_slot)) FERRIS_REFUSE("streams: a token shift goes with a read, a state and the step's positions and slots");
    const size_t smem = norm_w ? (size_t)width * sizeof(float) : 0;
    cudaStream_t s = (cudaStream_t)stream;
    // A thread's columns are taken one after another (a column's stores stand between its loads and the next column's),
    // so in a step of few rows a row is spread over as many threads as it has pairs of columns, up to 512; with many
    // rows the SMs are busy anyway and blocks of 256 move more (2,048 rows of 4 x 2,048: 74 against 100 us).
    const int wide = tokens < 256 ? 512 : 256;
    const dim3 grid(tokens), block(width >= 1024 ? wide : (width >= 512 ? 256 : 128));
    if (dtype == FERRIS_F32) {
        int e_ = ferris_allow_dynamic_smem((const void*)streams_step_kernel<float>, smem);
        if (e_ != FERRIS_OK) return e_;
        ferris_launch(streams_step_kernel<float>, grid, block, smem, s, xs, y, mix, out_w, in_w, norm_w, eps, (float*)out, streams, width, shift, shift_state, positions, seq_state_slot);
    } else if (dtype == FERRIS_BF16) {
        int e_ = ferris_allow_dynamic_smem((const void*)streams_step_kernel<bf16>, smem);
        if (e_ != FERRIS_OK) return e_;
        ferris_launch(streams_step_kernel<bf16>, grid, block, smem, s, xs, y, mix, out_w, in_w, norm_w, eps, (bf16*)out, streams, width, shift, shift_state, positions, seq_state_slot);
    } else
        FERRIS_REFUSE("streams: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}

// x, out: [tokens, width] of `dtype` (out must not be x); shift: fp32 [width]; state: fp32 [slots, width].
FERRIS_API int ferris_token_shift(const void* x, void* out, int dtype, const float* shift, float* state,
                                  const int* token_seq, const int* positions, const int* seq_q_start,
                                  const int* seq_start_pos, const int* seq_state_slot, int tokens, int seqs, int width,
                                  int advance, int single_tokens, void* stream) {
    if (tokens <= 0 || seqs <= 0) return FERRIS_OK;
    if (width <= 0 || !state || !shift) FERRIS_REFUSE("token shift: width %d, or no state or weights", width);
    if (x == out) FERRIS_REFUSE("token shift: input and output must differ");
    const int threads = width >= 256 ? 256 : ((width + 31) / 32) * 32;
    const int tiles = (width + threads - 1) / threads;
    if (tiles > 65535) FERRIS_REFUSE("token shift: %d columns are more than one launch takes", width);
    cudaStream_t s = (cudaStream_t)stream;
    const int single = (single_tokens && advance && tokens == seqs) ? 1 : 0;
    const dim3 block(threads), grid_a(tokens, tiles), grid_b(seqs, tiles);
    if (dtype == FERRIS_F32) {
        ferris_launch(token_shift_apply_kernel<float>, grid_a, block, 0, s, (const float*)x, (float*)out, shift, state, token_seq,
                      positions, seq_start_pos, seq_state_slot, width, single);
        if (advance && !single)
            ferris_launch(token_shift_advance_kernel<float>, grid_b, block, 0, s, (const float*)x, state, seq_q_start, seq_state_slot, width);
    } else if (dtype == FERRIS_BF16) {
        ferris_launch(token_shift_apply_kernel<bf16>, grid_a, block, 0, s, (const bf16*)x, (bf16*)out, shift, state, token_seq,
                      positions, seq_start_pos, seq_state_slot, width, single);
        if (advance && !single)
            ferris_launch(token_shift_advance_kernel<bf16>, grid_b, block, 0, s, (const bf16*)x, state, seq_q_start, seq_state_slot, width);
    } else
        FERRIS_REFUSE("token shift: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}

// h fp32 [tokens, width] += (accumulate) or = coef * sum_b rmsnorm(y_b) * w_b; y_b fp32 [tokens, width], w_b fp32 [width];
// 1..4 branches.
FERRIS_API int ferris_branch_norm_sum(const float* const* ys, const float* const* ws, int branches, float coef, float eps,
                                      float* h, int tokens, int width, int accumulate, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (branches < 1 || branches > 4 || width <= 0) FERRIS_REFUSE("branch norm: %d branches of %d", branches, width);
    Branches br = {};
    br.n = branches;
    for (int b = 0; b < branches; ++b) br.y[b] = ys[b], br.w[b] = ws[b];
    ferris_launch(branch_norm_sum_kernel, dim3(tokens), dim3(width >= 1024 ? 256 : 128), 0, (cudaStream_t)stream, br, coef, eps, h, width, accumulate);
    FERRIS_LAUNCH_CHECK();
}

// q (null: no queries): rows ldq apart of heads x (dim + rot); dkv (null: no keys): rows lddkv apart of rank + rot; cq (null: no
// query latent): rows ldcq apart of q_rank, normed into cq_out.  cache: [rows, rank + rot] (one kv head: a cache row per
// slot); q_att: rows ldqa apart.  The norms share eps.
FERRIS_API int ferris_latent_prepare(const void* q, int ldq, const void* dkv, int lddkv, int dtype, const float* norm_w, float eps,
                                     const int* positions, const float* freq, const float* freq_lo, int rot_dims, int interleaved,
                                     const int* slot_mapping, void* cache, void* q_att, int ldqa, const void* cq, int ldcq,
                                     const float* cq_norm, void* cq_out, int ldcq_out, int q_rank, int tokens, int heads,
                                     int dim, int rot, int rank, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (heads <= 0 || dim < 0 || rot < 0 || rank <= 0) FERRIS_REFUSE("latent prepare: %d heads of %d + %d over a latent of %d", heads, dim, rot, rank);
    if (rot_dims < 0 || rot_dims > rot || (rot_dims & 1) || rot_dims > 512) FERRIS_REFUSE("latent prepare: %d of %d dimensions rotate (at most 512)", rot_dims, rot);
    if (rot_dims > 0 && !freq) FERRIS_REFUSE("latent prepare: no frequencies");
    if (!positions || (q && !q_att)) FERRIS_REFUSE("latent prepare: no positions, or no rows for the queries");
    if (dkv && (!slot_mapping || !cache || !norm_w)) FERRIS_REFUSE("latent prepare: no cache to write");
    if (cq && (!cq_norm || !cq_out || q_rank <= 0)) FERRIS_REFUSE("latent prepare: a query latent of %d", q_rank);
    if (!q && !dkv && !cq) return FERRIS_OK;
    const LatentArgs p = {q, dkv, cq, cq_out, cq_norm, norm_w, freq, freq_lo, positions, slot_mapping, cache, q_att,
                          ldq, lddkv, ldcq, ldcq_out, ldqa, q_rank, rot_dims, interleaved, heads, dim, rot, rank, eps};
    const dim3 grid(tokens, cq && (q || dkv) ? 2 : 1);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == FERRIS_F32)
        ferris_launch(latent_prepare_kernel<float>, grid, dim3(128), 0, s, p);
    else if (dtype == FERRIS_BF16)
        ferris_launch(latent_prepare_kernel<bf16>, grid, dim3(128), 0, s, p);
    else
        FERRIS_REFUSE("latent prepare: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}

// x: [tokens, ...] with head h's K inputs at column h * hsx of rows ldx apart; w: [heads, K, N]; out likewise with hso,
// ldo; gate (may be null): [tokens, ...] rows ldg apart, one number per head.
FERRIS_API int ferris_head_gemm(const void* x, int ldx, int hsx, const void* w, void* out, int ldo, int hso,
                                const void* gate, int ldg, int dtype, int tokens, int heads, int K, int N, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (heads <= 0 || heads > 65535 || K <= 0 || N <= 0) FERRIS_REFUSE("head gemm: %d heads of %d x %d", heads, K, N);
    const size_t smem = ((size_t)HG_TOKENS * K + (size_t)(HG_PARTS - 1) * HG_TOKENS * HG_COLS) * sizeof(float);
    if (smem > 200 * 1024) FERRIS_REFUSE("head gemm: %d inputs a head are more than shared memory holds", K);
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == FERRIS_BF16 && tokens >= HM_MIN_TOKENS && K % 8 == 0 && N % 8 == 0 && ldx % 8 == 0 && hsx % 8 == 0 && ldo % 2 == 0 &&
        hso % 2 == 0 && (((uintptr_t)x | (uintptr_t)w) & 15) == 0 && ((uintptr_t)out & 3) == 0) {
        ferris_launch(head_gemm_mma_kernel, dim3((tokens + HM_TOKENS - 1) / HM_TOKENS, heads, (N + HM_COLS - 1) / HM_COLS), dim3(HM_THREADS), 0,
                      s, (const bf16*)x, ldx, hsx, (const bf16*)w, (bf16*)out, ldo, hso, (const bf16*)gate, ldg, tokens, K, N);
        FERRIS_LAUNCH_CHECK();
    }
    const dim3 grid((tokens + HG_TOKENS - 1) / HG_TOKENS, heads, (N + HG_COLS - 1) / HG_COLS), block(HG_THREADS);
    if (dtype == FERRIS_F32) {
        int e_ = ferris_allow_dynamic_smem((const void*)head_gemm_kernel<float>, smem);
        if (e_ != FERRIS_OK) return e_;
        ferris_launch(head_gemm_kernel<float>, grid, block, smem, s, (const float*)x, ldx, hsx, (const float*)w, (float*)out, ldo, hso,
                      (const float*)gate, ldg, tokens, K, N);
    } else if (dtype == FERRIS_BF16) {
        int e_ = ferris_allow_dynamic_smem((const void*)head_gemm_kernel<bf16>, smem);
        if (e_ != FERRIS_OK) return e_;
        ferris_launch(head_gemm_kernel<bf16>, grid, block, smem, s, (const bf16*)x, ldx, hsx, (const bf16*)w, (bf16*)out, ldo, hso,
                      (const bf16*)gate, ldg, tokens, K, N);
    } else
        FERRIS_REFUSE("head gemm: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}
