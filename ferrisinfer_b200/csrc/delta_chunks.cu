// The delta rule with a decay per key channel over portions of prompts, sixteen tokens at a time.
//
// Per (request, head), with rows r of S as key channels, d_t[r] <= 0 the logarithm of row r's decay at token t:
//     S <- diag(exp(d_t)) S;  u_t = b_t (v_t - S^T k_t);  S <- S + k_t u_t^T;  o_t = S^T q_t
// Walking the tokens one by one is a chain of dependent steps.  A chunk of C = 16 tokens has a closed form instead (the
// compact form of a product of rank-one corrections; Bischof and Van Loan's WY representation is its ancestor).  With
// L_t = d_1 + .. + d_t inside the chunk and S_0 the state at its start,
//     D_t = (k_t exp(L_t))^T S_0,   E_t = (q_t exp(L_t))^T S_0
//     A_ti = sum_r k_t k_i exp(L_t - L_i)  (i < t),   B_ti = sum_r q_t k_i exp(L_t - L_i)  (i <= t)
//     u_t = b_t (v_t - D_t - sum_(i<t) A_ti u_i)   i.e.  u = M (v - D),  M = (I + diag(b) A)^-1 diag(b)
//     o_t = E_t + sum_(i<=t) B_ti u_i
//     S_C = diag(exp(L_C)) S_0 + sum_i (k_i exp(L_C - L_i)) u_i^T
// Every exponent is of a difference that is not positive, so nothing overflows however fast a channel forgets, and the state
// moves on as S + (expm1(L_C) S + ..): a decay close to one is never rounded to 24 bits.  All of it is fp32.
//
// Two kernels.  What does not depend on the state (k_t exp(L_t), q_t exp(L_t), k_i exp(L_C - L_i), M, B, expm1(L_C)) is formed
// for all chunks side by side, a block per (chunk, head).  Then a block per (request, head, run of columns of S) walks the
// chunks: as in gated_recurrence.cu a few lanes share a column and hold eight rows each; here the sixteen tokens' products
// with S_0 are independent of one another, their sums over the lanes are reduced together (a lane ends with a token's sum, in
// 16 + 8 + .. exchanges instead of 16 x log2), and only the 16 x 16 products with M and B tie the tokens together.  The next
// chunk's rows come in by asynchronous copies meanwhile.
//
// For bf16 activations the walk runs on tensor cores: a block takes sixteen columns, its eight warps share the rows of S, and
// D^T = S_0^T K^T, E^T = S_0^T Q^T and the sum over the writes are products of tf32 fragments with fp32 sums.  Each operand x is
// cut into its leading eleven bits and the rest, and the products big x big, big x rest and rest x big are added, which keeps 21
// bits and more of every product; the state itself is only ever added to in fp32 outside the fragments' accumulators.
#include <math.h>

#include "common.cuh"

namespace {

constexpr int DC_TOKENS = 16;
constexpr int DC_THREADS = 128;
constexpr int DC_PREP_THREADS = 256;
constexpr int DC_KPL = 8;     // rows of the state that a lane holds
constexpr int DC_PITCH = 20;  // floats between the rows of 16 x 16 matrices in shared memory: rows start in different banks

// What a chunk of a head hands to the walk, in one piece of memory that a stage of shared memory takes as it is: kt, qt, kh
// [16][dim + 8], the products' rows (the pitch keeps the fragments' reads in different banks); dm [dim]; mm, bm [16][20].  Tokens
// beyond a chunk's last are zeros.  The place of a chunk is (its first row) / 16 + its request's index in the step, which no two
// chunks share.
__host__ __device__ constexpr int dc_pitch(int dim) { return dim + 8; }
__host__ __device__ constexpr int dc_stage_floats(int dim) { return 3 * DC_TOKENS * dc_pitch(dim) + dim + 2 * DC_TOKENS * DC_PITCH; }
struct DeltaStage {
    float *kt, *qt, *kh, *dm, *mm, *bm;
};
__device__ __forceinline__ DeltaStage dc_stage(float* base, int dim) {
    DeltaStage st;
    st.kt = base, st.qt = st.kt + DC_TOKENS * dc_pitch(dim), st.kh = st.qt + DC_TOKENS * dc_pitch(dim);
    st.dm = st.kh + DC_TOKENS * dc_pitch(dim), st.mm = st.dm + dim, st.bm = st.mm + DC_TOKENS * DC_PITCH;
    return st;
}
__device__ __forceinline__ float* dc_place(float* scratch, int first, int seq, int head, int heads, int dim) {
    return scratch + ((size_t)(first / DC_TOKENS + seq) * heads + head) * dc_stage_floats(dim);
}
// a stage's piece of memory into shared memory, 16 bytes at a time
__device__ __forceinline__ void dc_fetch(float* dst, const float* src, int floats, int threads) {
    const uint32_t to = (uint32_t)__cvta_generic_to_shared(dst);
    for (int x = threadIdx.x * 4; x < floats; x += threads * 4)
        asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(to + x * 4), "l"(src + x) : "memory");
}
__device__ __forceinline__ void dc_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void dc_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }

template <typename T>
__global__ void __launch_bounds__(DC_PREP_THREADS) delta_chunk_prepare_kernel(
    const T* q, int ldq, const T* k, int ldk, const float* z, int ldz, const float* __restrict__ rates, const float* beta,
    const float* qscale, const float* kscale, const int* __restrict__ seq_q_start, int chunks_max, int heads, int qk_heads, int dim,
    float* scratch) {
    extern __shared__ __align__(16) float dc_smem[];
    const int pitch = dim + 1;
    float* Ls = dc_smem;                     // [16][dim + 1]: logarithms, then their sums from the chunk's start
    float* Ks = Ls + DC_TOKENS * pitch;      // keys and queries with their factors
    float* Qs = Ks + DC_TOKENS * pitch;
    __shared__ float As[DC_TOKENS][DC_TOKENS + 1], bs[DC_TOKENS];
    pdl_wait();
    // (the walk is let in when this kernel's blocks end: its blocks would hold half of an SM's registers while they wait)
    const int seq = blockIdx.x / chunks_max, head = blockIdx.y;
    const int row0 = seq_q_start[seq], row1 = seq_q_start[seq + 1];
    const int first = row0 + (blockIdx.x % chunks_max) * DC_TOKENS;
    if (first >= row1) return;
    const int n = min(DC_TOKENS, row1 - first);
    const int qh = head / (heads / qk_heads);
    const float rate = rates[head];
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const DeltaStage st = dc_stage(dc_place(scratch, first, seq, head, heads, dim), dim);
    // an element (token, channel) a thread at a time: the next one is DC_PREP_THREADS further on
    const int step_t = DC_PREP_THREADS / dim, step_c = DC_PREP_THREADS - step_t * dim;
    const int t_mine = tid / dim, c_mine = tid - t_mine * dim;
    for (int t = t_mine, c = c_mine; t < DC_TOKENS;) {
        if (t < n) {
            const size_t row = (size_t)(first + t);
            Ls[t * pitch + c] = -ferris_softplus(z[row * ldz + (size_t)head * dim + c]) * rate;
            Ks[t * pitch + c] = to_float(k[row * ldk + (size_t)qh * dim + c]) * (kscale ? kscale[row * qk_heads + qh] : 1.0f);
            Qs[t * pitch + c] = to_float(q[row * ldq + (size_t)qh * dim + c]) * (qscale ? qscale[row * qk_heads + qh] : 1.0f);
        }
        t += step_t, c += step_c;
        if (c >= dim) c -= dim, ++t;
    }
    if (tid < DC_TOKENS) bs[tid] = tid < n ? beta[(size_t)(first + tid) * heads + head] : 0.0f;
    __syncthreads();
    for (int c = tid; c < dim; c += DC_PREP_THREADS) {
        float sum = 0.0f;
        for (int t = 0; t < n; ++t) sum += Ls[t * pitch + c], Ls[t * pitch + c] = sum;
        st.dm[c] = expm1f(sum);
    }
    __syncthreads();
    for (int t = t_mine, c = c_mine; t < DC_TOKENS;) {
        const int at = t * dc_pitch(dim) + c;
        if (t < n) {
            const float L = Ls[t * pitch + c], e = expf(L), kv = Ks[t * pitch + c];
            st.kt[at] = kv * e;
            st.qt[at] = Qs[t * pitch + c] * e;
            st.kh[at] = kv * expf(Ls[(n - 1) * pitch + c] - L);
        } else {
            st.kt[at] = st.qt[at] = st.kh[at] = 0.0f;
        }
        t += step_t, c += step_c;
        if (c >= dim) c -= dim, ++t;
    }
    constexpr float LOG2E = 1.4426950408889634f;
    // a warp takes tokens w and 15 - w: seventeen pairs each
    for (int half = 0; half < 2; ++half) {
        const int t = half ? DC_TOKENS - 1 - warp : warp;
        if (t >= n) {
            if (lane < DC_TOKENS) st.bm[t * DC_PITCH + lane] = 0.0f;
            continue;
        }
        float l[8], kv[8], qv[8];  // the token's row, a lane's channels lane, lane + 32, ..
#pragma unroll
        for (int j = 0; j < 8; ++j) {
            const int c = lane + 32 * j;
            l[j] = kv[j] = qv[j] = 0.0f;
            if (c < dim) l[j] = Ls[t * pitch + c], kv[j] = Ks[t * pitch + c], qv[j] = Qs[t * pitch + c];
        }
        for (int i = 0; i <= t; ++i) {
            float a = 0.0f, b = 0.0f;
#pragma unroll
            for (int j = 0; j < 8; ++j) {
                const int c = lane + 32 * j;
                if (32 * j < dim && c < dim) {
                    const float e = exp2f((l[j] - Ls[i * pitch + c]) * LOG2E) * Ks[i * pitch + c];
                    a = fmaf(kv[j], e, a), b = fmaf(qv[j], e, b);
                }
            }
            // both sums at once: the lower lanes end with a's, the upper ones with b's
            const bool upper = lane & 16;
            float sum = (upper ? b : a) + __shfl_xor_sync(0xffffffffu, upper ? a : b, 16);
#pragma unroll
            for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
            if (lane == 0) As[t][i] = sum;
            if (lane == 16) st.bm[t * DC_PITCH + i] = sum;
        }
        if (lane > t && lane < DC_TOKENS) st.bm[t * DC_PITCH + lane] = 0.0f;
    }
    __syncthreads();
    if (tid < DC_TOKENS) {  // a column of M each: M_tj = b_t (delta_tj - sum_(i<t) A_ti M_ij)
        float m[DC_TOKENS];
#pragma unroll
        for (int t = 0; t < DC_TOKENS; ++t) {
            float acc = t == tid ? 1.0f : 0.0f;
            if (t < n) {
#pragma unroll
                for (int i = 0; i < t; ++i) acc = fmaf(-As[t][i], m[i], acc);
                m[t] = bs[t] * acc;
            } else {
                m[t] = 0.0f;
            }
            st.mm[t * DC_PITCH + tid] = m[t];
        }
    }
}

// The sums over the LANES lanes of a column of sixteen numbers a lane: afterwards lane `sub` holds those of tokens
// sub * PER .. (LANES <= 16), or that of token sub / 2 (LANES = 32), in the first elements of x.
template <int LANES>
__device__ __forceinline__ void reduce_tokens(float (&x)[DC_TOKENS], int sub) {
    int width = DC_TOKENS;
#pragma unroll
    for (int o = LANES / 2; o > 0; o >>= 1) {
        if (width > 1) {
            width >>= 1;
            const bool upper = sub & o;
#pragma unroll
            for (int j = 0; j < DC_TOKENS / 2; ++j) {
                if (j < width) {
                    const float keep = upper ? x[j + width] : x[j], give = upper ? x[j] : x[j + width];
                    x[j] = keep + __shfl_xor_sync(0xffffffffu, give, o);
                }
            }
        } else {
            x[0] += __shfl_xor_sync(0xffffffffu, x[0], o);
        }
    }
}

template <typename T, int LANES>
__global__ void __launch_bounds__(DC_THREADS) delta_chunk_walk_kernel(
    float* scratch, const T* v, int ldv, float* __restrict__ out, int ldo, float* state, const int* __restrict__ seq_q_start,
    const int* __restrict__ seq_state_slot, int heads, int dim, int vdim, int write_state) {
    constexpr int COLS = DC_THREADS / LANES;  // columns of a block
    constexpr int PER = LANES >= DC_TOKENS ? 1 : DC_TOKENS / LANES;  // tokens whose sums a lane ends with
    extern __shared__ __align__(16) float dc_smem[];
    __shared__ __align__(16) float ws[COLS][DC_PITCH], us[COLS][DC_PITCH];
    pdl_wait();
    pdl_launch_dependents();
    const int seq = blockIdx.x, head = blockIdx.y, tid = threadIdx.x;
    const int sub = tid % LANES, cl = tid / LANES;
    const int col = blockIdx.z * COLS + cl;
    const bool active = col < vdim;
    const int row0 = seq_q_start[seq], row1 = seq_q_start[seq + 1];
    if (row1 <= row0) return;
    float* S = state + (((size_t)seq_state_slot[seq] * heads + head) * vdim + (active ? col : 0)) * (size_t)dim;
    float s[DC_KPL];
#pragma unroll
    for (int g = 0; g < 2; ++g) {
        const int r = (g * LANES + sub) * 4;
        float4 x = make_float4(0.0f, 0.0f, 0.0f, 0.0f);
        if (active && r < dim) x = *reinterpret_cast<const float4*>(S + r);
        s[4 * g] = x.x, s[4 * g + 1] = x.y, s[4 * g + 2] = x.z, s[4 * g + 3] = x.w;
    }
    const int mine = LANES == 32 ? sub >> 1 : sub * PER;  // the first token whose sums this lane ends with
    const bool writes = LANES != 32 || !(sub & 1);
    // the lane's two runs of four rows; a run beyond the head's size reads rows that its zero state does not feel, and its sums
    // over the writes are never used
    const int floats = dc_stage_floats(dim), pitch = dc_pitch(dim);
    const bool has[2] = {4 * sub < dim, 4 * (LANES + sub) < dim};
    const int r0 = has[0] ? 4 * sub : 0, r1 = has[1] ? 4 * (LANES + sub) : 0;
    auto fetch = [&](int first, int buf) {
        if (first < row1) dc_fetch(dc_smem + buf * floats, dc_place(scratch, first, seq, head, heads, dim), floats, DC_THREADS);
        dc_commit();
    };
    T pv[PER];
    auto request_v = [&](int first) {
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            const int t = first + mine + j;
            pv[j] = from_float<T>(0.0f);
            if (t < row1 && active) pv[j] = v[(size_t)t * ldv + (size_t)head * vdim + col];
        }
    };
    fetch(row0, 0);
    request_v(row0);
    int buf = 0;
    for (int first = row0; first < row1; first += DC_TOKENS, buf ^= 1) {
        fetch(first + DC_TOKENS, buf ^ 1);
        float vv[PER];
#pragma unroll
        for (int j = 0; j < PER; ++j) vv[j] = to_float(pv[j]);
        request_v(first + DC_TOKENS);
        dc_wait<1>();
        __syncthreads();
        const DeltaStage st = dc_stage(dc_smem + buf * floats, dim);
        float D[DC_TOKENS], E[DC_TOKENS];
#pragma unroll
        for (int t = 0; t < DC_TOKENS; ++t) {
            const float4 a = *reinterpret_cast<const float4*>(st.kt + t * pitch + r0);
            const float4 b = *reinterpret_cast<const float4*>(st.kt + t * pitch + r1);
            D[t] = fmaf(a.x, s[0], fmaf(a.y, s[1], fmaf(a.z, s[2], a.w * s[3])));
            D[t] = fmaf(b.x, s[4], fmaf(b.y, s[5], fmaf(b.z, s[6], fmaf(b.w, s[7], D[t]))));
            const float4 c = *reinterpret_cast<const float4*>(st.qt + t * pitch + r0);
            const float4 e = *reinterpret_cast<const float4*>(st.qt + t * pitch + r1);
            E[t] = fmaf(c.x, s[0], fmaf(c.y, s[1], fmaf(c.z, s[2], c.w * s[3])));
            E[t] = fmaf(e.x, s[4], fmaf(e.y, s[5], fmaf(e.z, s[6], fmaf(e.w, s[7], E[t]))));
        }
        reduce_tokens<LANES>(D, sub);
        reduce_tokens<LANES>(E, sub);
#pragma unroll
        for (int j = 0; j < PER; ++j)
            if (writes) ws[cl][mine + j] = vv[j] - D[j];
        __syncwarp();
        float x[DC_TOKENS];
#pragma unroll
        for (int i = 0; i < DC_TOKENS; i += 4) {
            const float4 f = *reinterpret_cast<const float4*>(&ws[cl][i]);
            x[i] = f.x, x[i + 1] = f.y, x[i + 2] = f.z, x[i + 3] = f.w;
        }
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            float u0 = 0.0f, u1 = 0.0f;
#pragma unroll
            for (int i = 0; i < DC_TOKENS; i += 4) {
                const float4 m = *reinterpret_cast<const float4*>(st.mm + (mine + j) * DC_PITCH + i);
                u0 = fmaf(m.x, x[i], u0), u1 = fmaf(m.y, x[i + 1], u1), u0 = fmaf(m.z, x[i + 2], u0), u1 = fmaf(m.w, x[i + 3], u1);
            }
            if (writes) us[cl][mine + j] = u0 + u1;
        }
        __syncwarp();
#pragma unroll
        for (int i = 0; i < DC_TOKENS; i += 4) {
            const float4 f = *reinterpret_cast<const float4*>(&us[cl][i]);
            x[i] = f.x, x[i + 1] = f.y, x[i + 2] = f.z, x[i + 3] = f.w;
        }
#pragma unroll
        for (int j = 0; j < PER; ++j) {
            float o0 = E[j], o1 = 0.0f;
#pragma unroll
            for (int i = 0; i < DC_TOKENS; i += 4) {
                const float4 m = *reinterpret_cast<const float4*>(st.bm + (mine + j) * DC_PITCH + i);
                o0 = fmaf(m.x, x[i], o0), o1 = fmaf(m.y, x[i + 1], o1), o0 = fmaf(m.z, x[i + 2], o0), o1 = fmaf(m.w, x[i + 3], o1);
            }
            const int t = first + mine + j;
            if (writes && active && t < row1) out[(size_t)t * ldo + (size_t)head * vdim + col] = o0 + o1;
        }
        float acc[DC_KPL];
#pragma unroll
        for (int i = 0; i < DC_KPL; ++i) acc[i] = 0.0f;
#pragma unroll
        for (int t = 0; t < DC_TOKENS; ++t) {
            const float4 a = *reinterpret_cast<const float4*>(st.kh + t * pitch + r0);
            const float4 b = *reinterpret_cast<const float4*>(st.kh + t * pitch + r1);
            acc[0] = fmaf(a.x, x[t], acc[0]), acc[1] = fmaf(a.y, x[t], acc[1]), acc[2] = fmaf(a.z, x[t], acc[2]), acc[3] = fmaf(a.w, x[t], acc[3]);
            acc[4] = fmaf(b.x, x[t], acc[4]), acc[5] = fmaf(b.y, x[t], acc[5]), acc[6] = fmaf(b.z, x[t], acc[6]), acc[7] = fmaf(b.w, x[t], acc[7]);
        }
        const float4 m0 = *reinterpret_cast<const float4*>(st.dm + r0), m1 = *reinterpret_cast<const float4*>(st.dm + r1);
        if (has[0]) s[0] += fmaf(m0.x, s[0], acc[0]), s[1] += fmaf(m0.y, s[1], acc[1]), s[2] += fmaf(m0.z, s[2], acc[2]), s[3] += fmaf(m0.w, s[3], acc[3]);
        if (has[1]) s[4] += fmaf(m1.x, s[4], acc[4]), s[5] += fmaf(m1.y, s[5], acc[5]), s[6] += fmaf(m1.z, s[6], acc[6]), s[7] += fmaf(m1.w, s[7], acc[7]);
        __syncthreads();  // the stage is read: the copies after next may overwrite it
    }
    dc_wait<0>();
    if (write_state && active) {
#pragma unroll
        for (int g = 0; g < 2; ++g) {
            const int r = (g * LANES + sub) * 4;
            if (r < dim) *reinterpret_cast<float4*>(S + r) = make_float4(s[4 * g], s[4 * g + 1], s[4 * g + 2], s[4 * g + 3]);
        }
    }
}

// ------------------------------------------------------------------------------------------ the walk on tensor cores
constexpr int DM_COLS = 16, DM_STAGES = 3, DM_WARPS = 8, DM_THREADS = 32 * DM_WARPS;

__device__ __forceinline__ void split_tf32(float x, uint32_t& big, uint32_t& rest) {
    big = __float_as_uint(x) & 0xffffe000u;
    rest = __float_as_uint(x - __uint_as_float(big));
}
__device__ __forceinline__ void mma_tf32_1688(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k8.row.col.f32.tf32.tf32.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}

// TILES: eight-row pieces of S that a warp holds at most (warp w's are w, w + 8, ..); dim a multiple of eight.
template <typename T, int TILES>
__global__ void __launch_bounds__(DM_THREADS) delta_chunk_walk_mma_kernel(
    float* scratch, const T* v, int ldv, float* __restrict__ out, int ldo, float* state, const int* __restrict__ seq_q_start,
    const int* __restrict__ seq_state_slot, int heads, int dim, int vdim, int write_state) {
    extern __shared__ __align__(16) float dc_smem[];
    __shared__ __align__(16) float pd[DM_WARPS][DM_COLS][DC_PITCH], pe[DM_WARPS][DM_COLS][DC_PITCH];
    __shared__ __align__(16) float ws[DM_COLS][DC_PITCH], us[DM_COLS][DC_PITCH];
    pdl_wait();
    pdl_launch_dependents();
    const int seq = blockIdx.x, head = blockIdx.y, col0 = blockIdx.z * DM_COLS, tid = threadIdx.x;
    const int warp = tid >> 5, lane = tid & 31, g = lane >> 2, t4 = lane & 3;
    const int row0 = seq_q_start[seq], row1 = seq_q_start[seq + 1];
    if (row1 <= row0) return;
    const int pitch = dc_pitch(dim), floats = dc_stage_floats(dim), tiles = dim >> 3;
    float* S = state + (((size_t)seq_state_slot[seq] * heads + head) * vdim + col0) * (size_t)dim;
    // S^T as an accumulator fragment: [0], [1]: column g, rows 8 j + 2 t4, + 1; [2], [3]: column g + 8.  The same registers are an A
    // fragment whose inner index is permuted (slot t4 is row 2 t4, slot t4 + 4 row 2 t4 + 1); B reads its rows the same way.
    float s[TILES][4];
#pragma unroll
    for (int j = 0; j < TILES; ++j) {
        const int tile = warp + DM_WARPS * j, r = 8 * tile + 2 * t4;
#pragma unroll
        for (int a = 0; a < 2; ++a) {
            float2 x = make_float2(0.0f, 0.0f);
            if (tile < tiles && col0 + g + 8 * a < vdim) x = *reinterpret_cast<const float2*>(S + (size_t)(g + 8 * a) * dim + r);
            s[j][2 * a] = x.x, s[j][2 * a + 1] = x.y;
        }
    }
    auto fetch = [&](int first, int stage) {
        if (first < row1) dc_fetch(dc_smem + stage * floats, dc_place(scratch, first, seq, head, heads, dim), floats, DM_THREADS);
        dc_commit();
    };
    const int cl = tid >> 4, tk = tid & 15;  // this thread's column and token between the products
    const bool active = col0 + cl < vdim;
    T pv;
    auto request_v = [&](int first) {
        pv = from_float<T>(0.0f);
        if (first + tk < row1 && active) pv = v[(size_t)(first + tk) * ldv + (size_t)head * vdim + col0 + cl];
    };
    fetch(row0, 0);
    fetch(row0 + DC_TOKENS, 1);
    request_v(row0);
    int stage = 0;
    for (int first = row0; first < row1; first += DC_TOKENS) {
        dc_wait<1>();
        __syncthreads();  // the stage is there; everyone is done with the one before, which the next copies overwrite
        fetch(first + 2 * DC_TOKENS, stage == 0 ? 2 : stage - 1);
        const float vv = to_float(pv);
        request_v(first + DC_TOKENS);
        const DeltaStage st = dc_stage(dc_smem + stage * floats, dim);
        // D^T and E^T over the warp's rows: two token tiles each, the small products in accumulators of their own
        float D[2][4], Dr[2][4], E[2][4], Er[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) D[n][e] = Dr[n][e] = E[n][e] = Er[n][e] = 0.0f;
#pragma unroll
        for (int j = 0; j < TILES; ++j) {
            const int tile = warp + DM_WARPS * j;
            if (tile < tiles) {
                uint32_t ab[4], ar[4];
                split_tf32(s[j][0], ab[0], ar[0]), split_tf32(s[j][2], ab[1], ar[1]);
                split_tf32(s[j][1], ab[2], ar[2]), split_tf32(s[j][3], ab[3], ar[3]);
#pragma unroll
                for (int n = 0; n < 2; ++n) {
                    const int at = (8 * n + g) * pitch + 8 * tile + 2 * t4;
                    const float2 x = *reinterpret_cast<const float2*>(st.kt + at);
                    const float2 y = *reinterpret_cast<const float2*>(st.qt + at);
                    uint32_t xb0, xr0, xb1, xr1, yb0, yr0, yb1, yr1;
                    split_tf32(x.x, xb0, xr0), split_tf32(x.y, xb1, xr1);
                    split_tf32(y.x, yb0, yr0), split_tf32(y.y, yb1, yr1);
                    mma_tf32_1688(D[n], ab, xb0, xb1);
                    mma_tf32_1688(E[n], ab, yb0, yb1);
                    mma_tf32_1688(Dr[n], ab, xr0, xr1);
                    mma_tf32_1688(Er[n], ab, yr0, yr1);
                    mma_tf32_1688(Dr[n], ar, xb0, xb1);
                    mma_tf32_1688(Er[n], ar, yb0, yb1);
                }
            }
        }
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int a = 0; a < 2; ++a) {
                const int c = g + 8 * a, t = 8 * n + 2 * t4;
                *reinterpret_cast<float2*>(&pd[warp][c][t]) = make_float2(D[n][2 * a] + Dr[n][2 * a], D[n][2 * a + 1] + Dr[n][2 * a + 1]);
                *reinterpret_cast<float2*>(&pe[warp][c][t]) = make_float2(E[n][2 * a] + Er[n][2 * a], E[n][2 * a + 1] + Er[n][2 * a + 1]);
            }
        __syncthreads();
        float e = 0.0f, x = 0.0f;
#pragma unroll
        for (int q = 0; q < DM_WARPS; ++q) x += pd[q][cl][tk], e += pe[q][cl][tk];
        ws[cl][tk] = vv - x;
        __syncwarp();  // a column's sixteen threads are of one warp
        float u0 = 0.0f, u1 = 0.0f;  // u = M w
#pragma unroll
        for (int i = 0; i < DC_TOKENS; i += 4) {
            const float4 f = *reinterpret_cast<const float4*>(&ws[cl][i]);
            const float4 m = *reinterpret_cast<const float4*>(st.mm + tk * DC_PITCH + i);
            u0 = fmaf(m.x, f.x, u0), u1 = fmaf(m.y, f.y, u1), u0 = fmaf(m.z, f.z, u0), u1 = fmaf(m.w, f.w, u1);
        }
        us[cl][tk] = u0 + u1;
        __syncthreads();
        // the writes: S^T += U^T K over the chunk's tokens, formed apart from the state and added to it in fp32
        {
            uint32_t ub[2][4], ur[2][4];
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                split_tf32(us[g][8 * k + t4], ub[k][0], ur[k][0]), split_tf32(us[g + 8][8 * k + t4], ub[k][1], ur[k][1]);
                split_tf32(us[g][8 * k + t4 + 4], ub[k][2], ur[k][2]), split_tf32(us[g + 8][8 * k + t4 + 4], ub[k][3], ur[k][3]);
            }
#pragma unroll
            for (int j = 0; j < TILES; ++j) {
                const int tile = warp + DM_WARPS * j;
                if (tile < tiles) {
                    float acc[4] = {0.0f, 0.0f, 0.0f, 0.0f}, rest[4] = {0.0f, 0.0f, 0.0f, 0.0f};
#pragma unroll
                    for (int k = 0; k < 2; ++k) {
                        uint32_t b0, r0, b1, r1;
                        split_tf32(st.kh[(8 * k + t4) * pitch + 8 * tile + g], b0, r0);
                        split_tf32(st.kh[(8 * k + t4 + 4) * pitch + 8 * tile + g], b1, r1);
                        mma_tf32_1688(acc, ub[k], b0, b1);
                        mma_tf32_1688(rest, ub[k], r0, r1);
                        mma_tf32_1688(rest, ur[k], b0, b1);
                    }
                    const float2 m = *reinterpret_cast<const float2*>(st.dm + 8 * tile + 2 * t4);
                    s[j][0] += fmaf(m.x, s[j][0], acc[0] + rest[0]), s[j][1] += fmaf(m.y, s[j][1], acc[1] + rest[1]);
                    s[j][2] += fmaf(m.x, s[j][2], acc[2] + rest[2]), s[j][3] += fmaf(m.y, s[j][3], acc[3] + rest[3]);
                }
            }
        }
        // o = E + B u
        {
            float o0 = e, o1 = 0.0f;
#pragma unroll
            for (int i = 0; i < DC_TOKENS; i += 4) {
                const float4 f = *reinterpret_cast<const float4*>(&us[cl][i]);
                const float4 m = *reinterpret_cast<const float4*>(st.bm + tk * DC_PITCH + i);
                o0 = fmaf(m.x, f.x, o0), o1 = fmaf(m.y, f.y, o1), o0 = fmaf(m.z, f.z, o0), o1 = fmaf(m.w, f.w, o1);
            }
            if (active && first + tk < row1) out[(size_t)(first + tk) * ldo + (size_t)head * vdim + col0 + cl] = o0 + o1;
        }
        stage = stage + 1 == DM_STAGES ? 0 : stage + 1;
    }
    dc_wait<0>();
    if (!write_state) return;
#pragma unroll
    for (int j = 0; j < TILES; ++j) {
        const int tile = warp + DM_WARPS * j, r = 8 * tile + 2 * t4;
#pragma unroll
        for (int a = 0; a < 2; ++a)
            if (tile < tiles && col0 + g + 8 * a < vdim)
                *reinterpret_cast<float2*>(S + (size_t)(g + 8 * a) * dim + r) = make_float2(s[j][2 * a], s[j][2 * a + 1]);
    }
}

template <typename T, int TILES>
int launch_walk_mma(float* scratch, const void* v, int ldv, float* out, int ldo, float* state, const int* seq_q_start,
                    const int* seq_state_slot, int seqs, int heads, int dim, int vdim, int write_state, cudaStream_t s) {
    const size_t smem = (size_t)DM_STAGES * dc_stage_floats(dim) * sizeof(float);
    const int rc = ferris_allow_dynamic_smem((const void*)delta_chunk_walk_mma_kernel<T, TILES>, smem);
    if (rc != FERRIS_OK) return rc;
    ferris_launch(delta_chunk_walk_mma_kernel<T, TILES>, dim3(seqs, heads, (vdim + DM_COLS - 1) / DM_COLS), dim3(DM_THREADS), smem, s, scratch,
                  (const T*)v, ldv, out, ldo, state, seq_q_start, seq_state_slot, heads, dim, vdim, write_state);
    FERRIS_LAUNCH_CHECK();
}

template <typename T, int LANES>
int launch_walk(float* scratch, const void* v, int ldv, float* out, int ldo, float* state, const int* seq_q_start,
                const int* seq_state_slot, int seqs, int heads, int dim, int vdim, int write_state, cudaStream_t s) {
    constexpr int COLS = DC_THREADS / LANES;
    const size_t smem = 2 * (size_t)dc_stage_floats(dim) * sizeof(float);
    const int rc = ferris_allow_dynamic_smem((const void*)delta_chunk_walk_kernel<T, LANES>, smem);
    if (rc != FERRIS_OK) return rc;
    ferris_launch(delta_chunk_walk_kernel<T, LANES>, dim3(seqs, heads, (vdim + COLS - 1) / COLS), dim3(DC_THREADS), smem, s, scratch,
                  (const T*)v, ldv, out, ldo, state, seq_q_start, seq_state_slot, heads, dim, vdim, write_state);
    FERRIS_LAUNCH_CHECK();
}

}  // namespace

// Floats of scratch that ferris_delta_chunks wants.
FERRIS_API long long ferris_delta_chunks_scratch(int tokens, int seqs, int heads, int dim) {
    return (long long)(tokens / DC_TOKENS + seqs + 1) * heads * dc_stage_floats(dim);
}

// Arguments as ferris_gated_recurrence with row decays (z, rates); dim a multiple of four, every pointer but v's on 16 bytes;
// longest: the most tokens a request brings.
FERRIS_API int ferris_delta_chunks(const void* q, int ldq, const void* k, int ldk, const void* v, int ldv, int dtype, const float* z,
                                   int ldz, const float* rates, const float* beta, const float* qscale, const float* kscale,
                                   float* out, int ldo, float* state, const int* seq_q_start, const int* seq_state_slot, int tokens,
                                   int seqs, int heads, int qk_heads, int dim, int vdim, int write_state, int longest, float* scratch,
                                   long long scratch_floats, void* stream) {
    if (seqs <= 0 || tokens <= 0) return FERRIS_OK;
    if (heads <= 0 || qk_heads <= 0 || heads % qk_heads) FERRIS_REFUSE("delta chunks: %d heads over %d q/k heads", heads, qk_heads);
    if (dim <= 0 || dim > 256 || dim % 4 || vdim <= 0) FERRIS_REFUSE("delta chunks: heads of %d x %d (multiples of 4, at most 256 rows)", dim, vdim);
    if (heads > 65535 || (vdim + 3) / 4 > 65535 || longest <= 0) FERRIS_REFUSE("delta chunks: too many heads or columns for one launch, or no length");
    if (!z || !rates || !beta || !scratch || scratch_floats < ferris_delta_chunks_scratch(tokens, seqs, heads, dim))
        FERRIS_REFUSE("delta chunks: decays, step sizes or scratch are missing");
    if (((uintptr_t)state | (uintptr_t)scratch) & 15) FERRIS_REFUSE("delta chunks: state and scratch must start on 16 bytes");
    const long long chunks_max = (longest + DC_TOKENS - 1) / DC_TOKENS;
    if (chunks_max * seqs > 2147483647LL) FERRIS_REFUSE("delta chunks: %d requests of up to %d tokens are more than one launch takes", seqs, longest);
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = 3 * (size_t)DC_TOKENS * (dim + 1) * sizeof(float);
    const dim3 grid((unsigned)(chunks_max * seqs), heads);
#define FERRIS_DC_GO(T)                                                                                                      \
    do {                                                                                                                     \
        int rc = ferris_allow_dynamic_smem((const void*)delta_chunk_prepare_kernel<T>, smem);                                 \
        if (rc != FERRIS_OK) return rc;                                                                                      \
        ferris_launch(delta_chunk_prepare_kernel<T>, grid, dim3(DC_PREP_THREADS), smem, s, (const T*)q, ldq, (const T*)k, ldk, z, \
                      ldz, rates, beta, qscale, kscale, seq_q_start, (int)chunks_max, heads, qk_heads, dim, scratch);               \
        if (dim <= 32) return launch_walk<T, 4>(scratch, v, ldv, out, ldo, state, seq_q_start, seq_state_slot, seqs, heads, dim, vdim, write_state, s); \
        if (dim <= 64) return launch_walk<T, 8>(scratch, v, ldv, out, ldo, state, seq_q_start, seq_state_slot, seqs, heads, dim, vdim, write_state, s); \
        if (dim <= 128) return launch_walk<T, 16>(scratch, v, ldv, out, ldo, state, seq_q_start, seq_state_slot, seqs, heads, dim, vdim, write_state, s); \
        return launch_walk<T, 32>(scratch, v, ldv, out, ldo, state, seq_q_start, seq_state_slot, seqs, heads, dim, vdim, write_state, s); \
    } while (0)
    if (dtype == FERRIS_BF16 && dim % 8 == 0) {
        int rc = ferris_allow_dynamic_smem((const void*)delta_chunk_prepare_kernel<bf16>, smem);
        if (rc != FERRIS_OK) return rc;
        ferris_launch(delta_chunk_prepare_kernel<bf16>, grid, dim3(DC_PREP_THREADS), smem, s, (const bf16*)q, ldq, (const bf16*)k, ldk, z,
                      ldz, rates, beta, qscale, kscale, seq_q_start, (int)chunks_max, heads, qk_heads, dim, scratch);
#define FERRIS_DM_GO(TILES) \
    return launch_walk_mma<bf16, TILES>(scratch, v, ldv, out, ldo, state, seq_q_start, seq_state_slot, seqs, heads, dim, vdim, write_state, s)
        if (dim <= 64) FERRIS_DM_GO(1);
        if (dim <= 128) FERRIS_DM_GO(2);
        FERRIS_DM_GO(4);
#undef FERRIS_DM_GO
    }
    if (dtype == FERRIS_F32) FERRIS_DC_GO(float);
    if (dtype == FERRIS_BF16) FERRIS_DC_GO(bf16);
#undef FERRIS_DC_GO
    FERRIS_REFUSE("delta chunks: unknown dtype %d", dtype);
}
