// The general attention over a bf16 cache on tensor cores, with the softmax's weights in 32-bit: head sizes of any multiple
// of eight up to 256 (the values' may differ, or lie in the keys), any page size, any grouping of heads, a window, a chunk or
// every key, pooled keys before the window or first tokens that it keeps, a soft cap, a sink, gates.  The formulas and arguments are those of attention_simt.cu.
//
// q . k is a product of bf16 numbers with fp32 sums, as exact as FMAs on the widened numbers.  The second product, weights
// times values, must not round the weights to bf16: a weight p is cut into three bf16 parts, p1 = bf16(p), p2 = bf16(p - p1),
// p3 = bf16(p - p1 - p2), whose sum is p to the last of its 24 bits, and the three products with the values meet in one fp32
// accumulator.  Scores, maximum, exponentials and sums are fp32 (powers of two: the scale carries log2 e).
//
// Two kernels.  Portions of prompts: a block takes 64 rows, the g query heads of one kv head for floor(64 / g) consecutive
// tokens, and walks the keys in tiles that asynchronous copies bring into shared memory one tile ahead; each of its four
// warps owns 16 rows.  Single tokens: a block takes one token, up to eight query heads of one kv head and a share of the
// keys; each of its four warps walks chunks of 16 keys of its own through a ring of asynchronous copies that only it reads
// (no block-wide barrier in the loop), and the four meet in shared memory at the end; the shares of a token are a cluster.
#include <math.h>

#include "attention_general.cuh"
#include "common.cuh"
#include "sm100.cuh"

namespace {

constexpr float LOG2E = 1.4426950408889634f;
constexpr int AR_THREADS = 128, AR_WARPS = 4, AR_ROWS = 64;

// 16 bytes into shared memory, or 16 zero bytes where the row is not there
__device__ __forceinline__ void copy16_or_zero(uint32_t dst, const void* src, bool there) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(there ? 16 : 0) : "memory");
}
__device__ __forceinline__ void ar_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N>
__device__ __forceinline__ void ar_wait() {
    asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory");
}

// The pair (a, b) as three packed pairs of bf16 whose sums are a and b.
__device__ __forceinline__ void split3(float a, float b, uint32_t& p1, uint32_t& p2, uint32_t& p3) {
    p1 = pack_bf16(a, b);
    a -= __uint_as_float(p1 << 16), b -= __uint_as_float(p1 & 0xffff0000u);
    p2 = pack_bf16(a, b);
    a -= __uint_as_float(p2 << 16), b -= __uint_as_float(p2 & 0xffff0000u);
    p3 = pack_bf16(a, b);
}

// Fragments of 16 query rows straight from global memory (a null row reads as zero); nks steps of 16 columns, the columns
// from d on are zero.
template <int KS>
__device__ __forceinline__ void load_q_rows(uint32_t (&qf)[KS][4], const bf16* row0, const bf16* row1, int d) {
    const int t = threadIdx.x & 3;
#pragma unroll
    for (int ks = 0; ks < KS; ++ks) {
        const int c = 16 * ks + 2 * t;
        qf[ks][0] = row0 && c < d ? *reinterpret_cast<const uint32_t*>(row0 + c) : 0u;
        qf[ks][1] = row1 && c < d ? *reinterpret_cast<const uint32_t*>(row1 + c) : 0u;
        qf[ks][2] = row0 && c + 8 < d ? *reinterpret_cast<const uint32_t*>(row0 + c + 8) : 0u;
        qf[ks][3] = row1 && c + 8 < d ? *reinterpret_cast<const uint32_t*>(row1 + c + 8) : 0u;
    }
}

struct AttentionArgs {
    const bf16* q;
    bf16* out;
    const bf16* k;
    const bf16* v;
    const int* tables;
    const int* token_seq;
    const int* positions;
    const float* sink;
    PooledKeys pk;  // every = keep = 0: none
    int ldq, ldo, max_blocks, tokens, nh, nkv, d, dv, page_size, window;
    float scale2;  // scale x log2 e; with a soft cap: cap x log2 e, and scale_cap = scale / cap
    float scale_cap;  // 0: no cap
    const bf16* gate;  // the heads' gates, rows ldgate apart (null: none)
    int ldgate;
    int values_in_keys;  // a value is the first dv elements of its key: the keys' tile serves both products, v is not read
};
// sigmoid of the gate of head h at token t
__device__ __forceinline__ float gate_of(const AttentionArgs& p, int t, int h) {
    return p.gate ? 1.0f / (1.0f + expf(-to_float(p.gate[(size_t)t * p.ldgate + h]))) : 1.0f;
}

__device__ __forceinline__ int page_of(const int* table, int j, int page_size, int pshift) {
    return table[pshift >= 0 ? (j >> pshift) : (j / page_size)];
}
__device__ __forceinline__ size_t row_of(int page, int head, int nkv, int j, int page_size, int pshift) {
    return ((size_t)page * nkv + head) * page_size + (pshift >= 0 ? (j & (page_size - 1)) : (j % page_size));
}
__device__ __forceinline__ int shift_of(int page_size) {
    return (page_size & (page_size - 1)) == 0 ? __ffs(page_size) - 1 : -1;
}

// One row pair's step of the running softmax over a tile of scores s (NT blocks of 8 keys; scaled, unseen ones -inf):
// scores become weights, the accumulators are brought to the new maximum.
template <int NT, int DT>
__device__ __forceinline__ void softmax_step(float (&s)[NT][4], float (&m)[2], float (&l)[2], float (&o)[DT][4]) {
    float alpha[2];
    bool moved = false;
#pragma unroll
    for (int a = 0; a < 2; ++a) {
        float best = -INFINITY;
#pragma unroll
        for (int n = 0; n < NT; ++n) best = fmaxf(best, fmaxf(s[n][2 * a], s[n][2 * a + 1]));
        best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 1));
        best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 2));
        const float m_new = fmaxf(m[a], best);
        const float base = m_new == -INFINITY ? 0.0f : m_new;  // a row that has seen nothing yet: every weight is 0
        alpha[a] = exp2f(m[a] - base);
        moved |= m_new != m[a];
        m[a] = m_new;
        float sum = 0.0f;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            s[n][2 * a] = exp2f(s[n][2 * a] - base);
            s[n][2 * a + 1] = exp2f(s[n][2 * a + 1] - base);
            sum += s[n][2 * a] + s[n][2 * a + 1];
        }
        l[a] = l[a] * alpha[a] + sum;
    }
    if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
        for (int n = 0; n < DT; ++n) o[n][0] *= alpha[0], o[n][1] *= alpha[0], o[n][2] *= alpha[1], o[n][3] *= alpha[1];
    }
}

// o += weights of 16 keys (blocks 2 kk and 2 kk + 1 of s) times their values (rows of pitch vp bytes from v_base).
template <int NT, int DT>
__device__ __forceinline__ void weights_times_values(float (&o)[DT][4], const float (&s)[NT][4], int kk, uint32_t v_base, int vp,
                                                     int dv) {
    const int lane = threadIdx.x & 31;
    uint32_t p[3][4];
    split3(s[2 * kk][0], s[2 * kk][1], p[0][0], p[1][0], p[2][0]);
    split3(s[2 * kk][2], s[2 * kk][3], p[0][1], p[1][1], p[2][1]);
    split3(s[2 * kk + 1][0], s[2 * kk + 1][1], p[0][2], p[1][2], p[2][2]);
    split3(s[2 * kk + 1][2], s[2 * kk + 1][3], p[0][3], p[1][3], p[2][3]);
    const uint32_t at = v_base + (uint32_t)(16 * kk + ((lane >> 3) & 1) * 8 + (lane & 7)) * vp + (lane >> 4) * 16;
    // four accumulators in turn, so that a part's product does not wait for the part's before it
#pragma unroll
    for (int n = 0; n < DT; n += 4) {
        if (8 * n < dv) {
            uint32_t b[2][4];
            ldmatrix_x4_trans(b[0], at + n * 16);
            ldmatrix_x4_trans(b[1], at + n * 16 + 32);
#pragma unroll
            for (int x = 0; x < 3; ++x) {
                mma_bf16_16816(o[n], p[x], b[0][0], b[0][1]);
                mma_bf16_16816(o[n + 1], p[x], b[0][2], b[0][3]);
                mma_bf16_16816(o[n + 2], p[x], b[1][0], b[1][1]);
                mma_bf16_16816(o[n + 3], p[x], b[1][2], b[1][3]);
            }
        }
    }
}

// ------------------------------------------------------------------------------------------ portions of prompts
// D: columns held for a head (64, 128, 256; d, dv <= D).  KT: keys to a tile.  The query fragments stay in registers up to
// D = 128 and come from shared memory beyond.
template <int D, int KT, bool POOL>
__global__ void __launch_bounds__(AR_THREADS, D <= 128 ? 3 : 2) attention_rows_kernel(const AttentionArgs p) {
    constexpr int KS = D / 16, DT = D / 8, NT = KT / 8;
    constexpr bool QREG = D <= 128;
    extern __shared__ __align__(16) uint8_t ar_smem[];
    constexpr int PITCH = (D + 8) * 2;  // bytes of a row: 16 more than the columns, so that eight rows lie in different banks
    const uint32_t base = smem_u32(ar_smem);
    constexpr uint32_t V_OFF = KT * PITCH, STAGE = 2 * KT * PITCH, Q_OFF = 2 * STAGE;
    pdl_wait();
    pdl_launch_dependents();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gq = lane >> 2, tq = lane & 3;
    const int g = p.nh / p.nkv, qt = AR_ROWS / g;
    const int hk = blockIdx.y;
    const int t_first = (gridDim.x - 1 - blockIdx.x) * qt;  // the last tokens, which see most keys, first
    const int t_end = min(t_first + qt, p.tokens);
    const int pshift = shift_of(p.page_size);
    const int d = p.d, dv = p.dv;
    const int nks = (d + 15) >> 4;

    // columns between d and the next multiple of 16 are zero on both sides
    if (d & 15) {
        for (int r = tid; r < 2 * KT; r += AR_THREADS)
            *reinterpret_cast<uint4*>(ar_smem + (r / KT) * STAGE + (r % KT) * PITCH + d * 2) = make_uint4(0u, 0u, 0u, 0u);
    }
    int rt[2], rpos[2], rseq[2];
    const bf16* qrow[2];
#pragma unroll
    for (int a = 0; a < 2; ++a) {
        const int r = 16 * warp + gq + 8 * a;
        rt[a] = r < qt * g ? t_first + r / g : p.tokens;
        const bool ok = rt[a] < t_end;
        rpos[a] = ok ? p.positions[rt[a]] : -1;
        rseq[a] = ok ? p.token_seq[rt[a]] : -1;
        qrow[a] = ok ? p.q + (size_t)rt[a] * p.ldq + (size_t)(hk * g + r % g) * d : nullptr;
    }
    uint32_t qf[QREG ? KS : 1][4];
    if constexpr (QREG) {
        load_q_rows<KS>(qf, qrow[0], qrow[1], d);
    } else {
        for (int x = tid; x < AR_ROWS * (D / 8); x += AR_THREADS) {
            const int r = x / (D / 8), c = x % (D / 8);
            const int t = r < qt * g ? t_first + r / g : p.tokens;
            uint4 u = make_uint4(0u, 0u, 0u, 0u);
            if (t < t_end && 8 * c < d)
                u = *reinterpret_cast<const uint4*>(p.q + (size_t)t * p.ldq + (size_t)(hk * g + r % g) * d + 8 * c);
            *reinterpret_cast<uint4*>(ar_smem + Q_OFF + r * PITCH + c * 16) = u;
        }
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    float o[DT][4];
#pragma unroll
    for (int n = 0; n < DT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.0f;

    const int seq_first = p.token_seq[t_first], seq_last = p.token_seq[t_end - 1];
    int ta = t_first;  // first token of the current request within the tile
    for (int sq = seq_first; sq <= seq_last; ++sq) {
        int tb = ta;  // its last token within the tile
        while (tb + 1 < t_end && p.token_seq[tb + 1] == sq) ++tb;
        const int pa = p.positions[ta], pb = p.positions[tb];
        const int kmin = first_key(pa, p.window);  // of the first token: no later token of the request sees an earlier key
        const int runs = POOL ? ahead_rows(p.pk, first_key(pb, p.window)) : 0;
        const int run_tiles = (runs + KT - 1) / KT;
        const int tiles = run_tiles + (pb - kmin + KT) / KT;
        const int* table = p.tables + (size_t)sq * p.max_blocks;
        const int* ptable = POOL ? p.pk.tables + (size_t)sq * p.pk.max_blocks : nullptr;
        constexpr int TPK = AR_THREADS / KT;  // threads that copy a key
        const int key = tid / TPK, part = tid % TPK;
        auto page_at = [&](int i) -> int {  // page of this thread's key in tile i, -1 if the tile does not hold it
            if (i >= tiles) return -1;
            if (POOL && i < run_tiles) {
                const int j = i * KT + key;
                return j < runs ? page_of(ptable, j, p.page_size, pshift) : -1;
            }
            const int j = kmin + (i - run_tiles) * KT + key;
            return j <= pb ? page_of(table, j, p.page_size, pshift) : -1;
        };
        auto fetch = [&](int i, int page) {
            if (i < tiles) {
                const bool run = POOL && i < run_tiles;
                const int j = run ? i * KT + key : kmin + (i - run_tiles) * KT + key;
                const bool there = page >= 0;
                const size_t row = there ? row_of(page, hk, p.nkv, j, p.page_size, pshift) : 0;
                const bf16* ks = (run ? reinterpret_cast<const bf16*>(p.pk.k) : p.k) + row * d;
                const bf16* vs = (run ? reinterpret_cast<const bf16*>(p.pk.v) : p.v) + row * dv;
                const uint32_t dst = base + (i & 1) * STAGE + key * PITCH;
                for (int c = part; c < (d >> 3); c += TPK) copy16_or_zero(dst + c * 16, ks + 8 * c, there);
                if (!p.values_in_keys)
                    for (int c = part; c < (dv >> 3); c += TPK) copy16_or_zero(dst + V_OFF + c * 16, vs + 8 * c, there);
            }
            ar_commit();
        };
        __syncthreads();  // the request before has been read (and, the first time, the zero columns and queries are in place)
        fetch(0, page_at(0));
        int next_page = page_at(1);
        int hi[2], lo[2], seen_runs[2];
#pragma unroll
        for (int a = 0; a < 2; ++a) {
            const bool mine = rseq[a] == sq;
            lo[a] = mine ? first_key(rpos[a], p.window) : 0;
            hi[a] = mine ? rpos[a] : -1;
            seen_runs[a] = POOL && mine ? ahead_rows(p.pk, lo[a]) : 0;
        }
        for (int i = 0; i < tiles; ++i) {
            fetch(i + 1, next_page);
            next_page = page_at(i + 2);
            ar_wait<1>();
            __syncthreads();
            const uint32_t kb = base + (i & 1) * STAGE;
            float s[NT][4];
#pragma unroll
            for (int n = 0; n < NT; ++n)
#pragma unroll
                for (int e = 0; e < 4; ++e) s[n][e] = 0.0f;
            const uint32_t k_at = kb + (uint32_t)((lane >> 4) * 8 + (lane & 7)) * PITCH + ((lane >> 3) & 1) * 16;
            const uint32_t q_at = base + Q_OFF + (uint32_t)(16 * warp + (lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + (lane >> 4) * 16;
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
                if (ks < nks) {
                    uint32_t af[4];
                    if constexpr (QREG) {
#pragma unroll
                        for (int e = 0; e < 4; ++e) af[e] = qf[ks][e];
                    } else {
                        ldmatrix_x4(af, q_at + ks * 32);
                    }
#pragma unroll
                    for (int n = 0; n < NT; n += 2) {
                        uint32_t b[4];
                        ldmatrix_x4(b, k_at + (uint32_t)(8 * n) * PITCH + ks * 32);
                        mma_bf16_16816(s[n], af, b[0], b[1]);
                        mma_bf16_16816(s[n + 1], af, b[2], b[3]);
                    }
                }
            }
            if (p.scale_cap > 0.0f) {
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[n][e] = tanhf(s[n][e] * p.scale_cap);
            }
            const bool run = POOL && i < run_tiles;
            const int j0 = run ? i * KT : kmin + (i - run_tiles) * KT;
            int from[2], to[2];  // of the tile's keys, those that the rows see
#pragma unroll
            for (int a = 0; a < 2; ++a) {
                from[a] = run ? 0 : lo[a] - j0;
                to[a] = (run ? seen_runs[a] - 1 : hi[a]) - j0;
            }
            const bool whole = from[0] <= 0 && from[1] <= 0 && to[0] >= KT - 1 && to[1] >= KT - 1;
            if (__all_sync(0xffffffffu, whole)) {
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) s[n][e] *= p.scale2;
            } else {
#pragma unroll
                for (int n = 0; n < NT; ++n)
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int c = 8 * n + 2 * tq + (e & 1);
                        s[n][e] = c >= from[e >> 1] && c <= to[e >> 1] ? s[n][e] * p.scale2 : -INFINITY;
                    }
            }
            softmax_step<NT, DT>(s, m, l, o);
#pragma unroll
            for (int kk = 0; kk < KT / 16; ++kk) weights_times_values<NT, DT>(o, s, kk, p.values_in_keys ? kb : kb + V_OFF, PITCH, dv);
            __syncthreads();  // the stage is read: the copies after next may overwrite it
        }
        ta = tb + 1;
    }
    ar_wait<0>();
#pragma unroll
    for (int a = 0; a < 2; ++a) {
        l[a] += __shfl_xor_sync(0xffffffffu, l[a], 1);
        l[a] += __shfl_xor_sync(0xffffffffu, l[a], 2);
        if (rt[a] >= t_end) continue;
        const int head = hk * g + (16 * warp + gq + 8 * a) % g;
        const float sink = p.sink ? exp2f(p.sink[head] * LOG2E - m[a]) : 0.0f;
        const float inv = gate_of(p, rt[a], head) / (l[a] + sink);
        bf16* orow = p.out + (size_t)rt[a] * p.ldo + (size_t)head * dv;
#pragma unroll
        for (int n = 0; n < DT; ++n) {
            const int c = 8 * n + 2 * tq;
            if (c < dv) *reinterpret_cast<uint32_t*>(orow + c) = pack_bf16(o[n][2 * a] * inv, o[n][2 * a + 1] * inv);
        }
    }
}

template <int D>
constexpr int rows_keys() { return D <= 128 ? 64 : 32; }
template <int D>
constexpr size_t rows_smem() {
    return (size_t)4 * rows_keys<D>() * (D + 8) * 2 + (D <= 128 ? 0 : (size_t)AR_ROWS * (D + 8) * 2);
}

// ------------------------------------------------------------------------------------------ single tokens
// A token's query heads of one kv head are few (a row group holds up to eight), so they stand on the narrow side of the
// fragments: S^T = K Q^T (16 keys x 8 heads), O^T = V^T P^T (16 value columns x 8 heads).  A chunk is 16 positions that begin
// at a multiple of 16, so that with FAST (heads of exactly D, pages of a multiple of 16) its keys lie in one piece of memory
// and one table look-up finds them.  A warp's chunks: the pooled runs' first, then the tokens', every fourth of the share.
// The shares of a token's keys (splits > 1) are a thread-block cluster, which merges them through its shared memory.
constexpr int AS_KEYS = 16, AS_ROWS = 8, AS_MAX_SPLITS = 8;
template <int D>
struct SingleStages {
    static constexpr int value = D <= 64 ? 4 : (D <= 128 ? 3 : 2);
};

template <int D, bool POOL, bool FAST>
__global__ void __launch_bounds__(AR_THREADS) attention_single_rows_kernel(const AttentionArgs p, int row_groups, int splits) {
    constexpr int KS = D / 16, MT = D / 16, STAGES = SingleStages<D>::value;
    constexpr int PITCH = (D + 8) * 2;
    constexpr uint32_t V_OFF = AS_KEYS * PITCH, STAGE = 2 * AS_KEYS * PITCH;
    extern __shared__ __align__(16) uint8_t ar_smem[];
    pdl_wait();
    pdl_launch_dependents();
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, gq = lane >> 2, tq = lane & 3;
    const int t = blockIdx.x, hk = blockIdx.y / row_groups, r0 = (blockIdx.y % row_groups) * AS_ROWS, split = blockIdx.z;
    const int g = p.nh / p.nkv, rows = min(AS_ROWS, g - r0);
    const int seq = p.token_seq[t], P = p.positions[t];
    const int pshift = shift_of(p.page_size);
    const int d = FAST ? D : p.d, dv = FAST ? D : p.dv;
    const int nks = FAST ? KS : (d + 15) >> 4;
    const int lo = first_key(P, p.window);
    const int pooled = POOL ? ahead_rows(p.pk, lo) : 0;
    const int run_chunks = (pooled + AS_KEYS - 1) / AS_KEYS;
    const int token_chunk = lo / AS_KEYS - run_chunks;  // chunk c >= run_chunks holds the tokens from 16 (c + token_chunk) on
    const int chunks_all = P / AS_KEYS - token_chunk + 1;
    const int per = (chunks_all + splits - 1) / splits;
    const int c_first = split * per + warp, c_end = min(chunks_all, split * per + per);
    const int* table = p.tables + (size_t)seq * p.max_blocks;
    const int* ptable = POOL ? p.pk.tables + (size_t)seq * p.pk.max_blocks : nullptr;

    uint8_t* mine = ar_smem + warp * STAGES * STAGE;
    const uint32_t ring = smem_u32(mine);
    if (!FAST && (d & 15)) {  // columns between d and the next multiple of 16 are zero on both sides
        for (int r = lane; r < STAGES * AS_KEYS; r += 32)
            *reinterpret_cast<uint4*>(mine + (r / AS_KEYS) * STAGE + (r % AS_KEYS) * PITCH + d * 2) = make_uint4(0u, 0u, 0u, 0u);
    }
    uint32_t qf[KS][2];
    {
        const bf16* row = p.q + (size_t)t * p.ldq + (size_t)(hk * g + r0 + gq) * d;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            const int c = 16 * ks + 2 * tq;
            qf[ks][0] = gq < rows && c < d ? *reinterpret_cast<const uint32_t*>(row + c) : 0u;
            qf[ks][1] = gq < rows && c + 8 < d ? *reinterpret_cast<const uint32_t*>(row + c + 8) : 0u;
        }
    }
    float m[2] = {-INFINITY, -INFINITY}, l[2] = {0.0f, 0.0f};
    float o[MT][4];
#pragma unroll
    for (int n = 0; n < MT; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.0f;

    // of chunk c (this warp's are c_first, c_first + 4, ...): its first position, and which of its 16 keys are seen
    auto first_of = [&](int c) -> int { return POOL && c < run_chunks ? c * AS_KEYS : (c + token_chunk) * AS_KEYS; };
    auto from_of = [&](int c) -> int { return POOL && c < run_chunks ? 0 : lo - first_of(c); };
    auto to_of = [&](int c) -> int { return (POOL && c < run_chunks ? pooled - 1 : P) - first_of(c); };
    const int key = FAST ? 0 : lane >> 1, part = lane & 1;
    auto page_at = [&](int c) -> int {
        if (c >= c_end || (!FAST && (key < from_of(c) || key > to_of(c)))) return -1;
        return page_of(POOL && c < run_chunks ? ptable : table, first_of(c) + key, p.page_size, pshift);
    };
    auto fetch = [&](int c, int stage, int page) {
        if (c < c_end) {
            const bool run = POOL && c < run_chunks, there = page >= 0;
            const size_t row = there ? row_of(page, hk, p.nkv, first_of(c) + key, p.page_size, pshift) : 0;
            const bf16* ks = (run ? reinterpret_cast<const bf16*>(p.pk.k) : p.k) + row * d;
            const bf16* vs = (run ? reinterpret_cast<const bf16*>(p.pk.v) : p.v) + row * dv;
            const uint32_t dst = ring + stage * STAGE;
            if constexpr (FAST) {  // 16 keys in one piece: a warp copies 512 bytes of it at a time
                const int from = from_of(c), to = to_of(c);
                constexpr int PIECES = D / 8;  // of a row
#pragma unroll
                for (int it = 0; it < AS_KEYS * PIECES / 32; ++it) {
                    const int x = it * 32 + lane, r = x / PIECES, col = x % PIECES;
                    const bool seen = there && r >= from && r <= to;
                    copy16_or_zero(dst + r * PITCH + col * 16, ks + 8 * x, seen);
                    copy16_or_zero(dst + V_OFF + r * PITCH + col * 16, vs + 8 * x, seen);
                }
            } else {
                for (int x = part; x < (d >> 3); x += 2) copy16_or_zero(dst + key * PITCH + x * 16, ks + 8 * x, there);
                if (!p.values_in_keys)
                    for (int x = part; x < (dv >> 3); x += 2) copy16_or_zero(dst + V_OFF + key * PITCH + x * 16, vs + 8 * x, there);
            }
        }
        ar_commit();
    };
    {
        int pages[STAGES - 1];
#pragma unroll
        for (int i = 0; i < STAGES - 1; ++i) pages[i] = page_at(c_first + AR_WARPS * i);
#pragma unroll
        for (int i = 0; i < STAGES - 1; ++i) fetch(c_first + AR_WARPS * i, i, pages[i]);
    }
    int next_page = page_at(c_first + AR_WARPS * (STAGES - 1));
    int stage = 0, fill = STAGES - 1;
    for (int c = c_first; c < c_end; c += AR_WARPS) {
        fetch(c + AR_WARPS * (STAGES - 1), fill, next_page);
        next_page = page_at(c + AR_WARPS * STAGES);
        ar_wait<STAGES - 1>();
        __syncwarp();
        const uint32_t kb = ring + stage * STAGE;
        float s[2][4];  // two accumulators, so that the products do not wait for one another
#pragma unroll
        for (int e = 0; e < 4; ++e) s[0][e] = 0.0f, s[1][e] = 0.0f;
        const uint32_t k_at = kb + (uint32_t)((lane & 7) + ((lane >> 3) & 1) * 8) * PITCH + (lane >> 4) * 16;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            if (ks < nks) {
                uint32_t a[4];
                ldmatrix_x4(a, k_at + ks * 32);
                mma_bf16_16816(s[ks & 1], a, qf[ks][0], qf[ks][1]);
            }
        }
        // keys gq and gq + 8 of the chunk against heads 2 tq and 2 tq + 1
        const int from = from_of(c), to = to_of(c);
        float w[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int at = gq + (e >> 1) * 8;
            float x = s[0][e] + s[1][e];
            if (p.scale_cap > 0.0f) x = tanhf(x * p.scale_cap);
            w[e] = at >= from && at <= to ? x * p.scale2 : -INFINITY;
        }
        float alpha[2];
        bool moved = false;
#pragma unroll
        for (int a = 0; a < 2; ++a) {
            float best = fmaxf(w[a], w[2 + a]);
            best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 4));
            best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 8));
            best = fmaxf(best, __shfl_xor_sync(0xffffffffu, best, 16));
            const float m_new = fmaxf(m[a], best);
            const float base = m_new == -INFINITY ? 0.0f : m_new;
            alpha[a] = exp2f(m[a] - base);
            moved |= m_new != m[a];
            m[a] = m_new;
            w[a] = exp2f(w[a] - base), w[2 + a] = exp2f(w[2 + a] - base);
            l[a] = l[a] * alpha[a] + (w[a] + w[2 + a]);
        }
        if (__any_sync(0xffffffffu, moved)) {
#pragma unroll
            for (int n = 0; n < MT; ++n) o[n][0] *= alpha[0], o[n][1] *= alpha[1], o[n][2] *= alpha[0], o[n][3] *= alpha[1];
        }
        uint32_t pw[3][2];
        split3(w[0], w[1], pw[0][0], pw[1][0], pw[2][0]);
        split3(w[2], w[3], pw[0][1], pw[1][1], pw[2][1]);
#pragma unroll
        for (int x = 0; x < 3; ++x) pw[x][0] = movmatrix_trans(pw[x][0]), pw[x][1] = movmatrix_trans(pw[x][1]);
        const uint32_t v_at = kb + (!FAST && p.values_in_keys ? 0 : V_OFF) + (uint32_t)((lane & 7) + (lane >> 4) * 8) * PITCH + ((lane >> 3) & 1) * 16;
#pragma unroll
        for (int n = 0; n < MT; n += 4) {  // four accumulators in turn
            if (16 * n < dv) {
                uint32_t a[4][4];
#pragma unroll
                for (int i = 0; i < 4; ++i) ldmatrix_x4_trans(a[i], v_at + (n + i) * 32);
#pragma unroll
                for (int x = 0; x < 3; ++x)
#pragma unroll
                    for (int i = 0; i < 4; ++i) mma_bf16_16816(o[n + i], a[i], pw[x][0], pw[x][1]);
            }
        }
        __syncwarp();  // the stage is read: the copy after next may overwrite it
        stage = stage + 1 == STAGES ? 0 : stage + 1;
        fill = fill + 1 == STAGES ? 0 : fill + 1;
    }
    ar_wait<0>();
    // the four warps meet: per warp and head its maximum, sum and weighted values
    float* meet = reinterpret_cast<float*>(ar_smem);
    const int stride = dv + 2;
    __syncthreads();
#pragma unroll
    for (int a = 0; a < 2; ++a) {
#pragma unroll
        for (int x = 4; x <= 16; x <<= 1) l[a] += __shfl_xor_sync(0xffffffffu, l[a], x);
        const int r = 2 * tq + a;
        if (r < rows) {
            float* e = meet + (size_t)(warp * rows + r) * stride;
            if (gq == 0) e[0] = m[a], e[1] = l[a];
#pragma unroll
            for (int n = 0; n < MT; ++n) {
                const int c = 16 * n + gq;
                if (c < dv) e[2 + c] = o[n][a];
                if (c + 8 < dv) e[2 + c + 8] = o[n][2 + a];
            }
        }
    }
    __syncthreads();
    for (int x = threadIdx.x; x < rows * dv; x += AR_THREADS) {
        const int r = x / dv, i = x - r * dv;
        float mm = -INFINITY;
#pragma unroll
        for (int w = 0; w < AR_WARPS; ++w) mm = fmaxf(mm, meet[(size_t)(w * rows + r) * stride]);
        float zz = 0.0f, acc = 0.0f;
#pragma unroll
        for (int w = 0; w < AR_WARPS; ++w) {
            const float* e = meet + (size_t)(w * rows + r) * stride;
            const float f = e[0] == -INFINITY ? 0.0f : exp2f(e[0] - mm);
            zz = fmaf(e[1], f, zz), acc = fmaf(e[2 + i], f, acc);
        }
        if (splits == 1) {
            const int head = hk * g + r0 + r;
            if (p.sink) zz += exp2f(p.sink[head] * LOG2E - mm);
            p.out[(size_t)t * p.ldo + (size_t)head * dv + i] = from_float<bf16>(acc / zz * gate_of(p, t, head));
        } else {
            float* e = meet + (size_t)(AR_WARPS * rows + r) * stride;
            if (i == 0) e[0] = mm, e[1] = zz;
            e[2 + i] = acc;
        }
    }
    if (splits == 1) return;
    // the shares of a token are the blocks of a cluster: each adds up its part of the outputs from all of them
    cluster_sync();
    const uint32_t shares = smem_u32(meet + (size_t)AR_WARPS * rows * stride);
    for (int x = split * AR_THREADS + threadIdx.x; x < rows * dv; x += splits * AR_THREADS) {
        const int r = x / dv, i = x - r * dv;
        const uint32_t at = shares + (uint32_t)(r * stride) * 4;
        float ms[AS_MAX_SPLITS], mm = -INFINITY;
#pragma unroll
        for (int w = 0; w < AS_MAX_SPLITS; ++w) {
            ms[w] = w < splits ? ld_peer_shared_f32(at, w) : -INFINITY;
            mm = fmaxf(mm, ms[w]);
        }
        float zz = 0.0f, acc = 0.0f;
#pragma unroll
        for (int w = 0; w < AS_MAX_SPLITS; ++w) {
            if (w < splits && ms[w] != -INFINITY) {
                const float f = exp2f(ms[w] - mm);
                zz = fmaf(ld_peer_shared_f32(at + 4, w), f, zz), acc = fmaf(ld_peer_shared_f32(at + 8 + 4 * i, w), f, acc);
            }
        }
        const int head = hk * g + r0 + r;
        if (p.sink) zz += exp2f(p.sink[head] * LOG2E - mm);
        p.out[(size_t)t * p.ldo + (size_t)head * dv + i] = from_float<bf16>(acc / zz * gate_of(p, t, head));
    }
    cluster_sync();  // nobody leaves while a peer may still read its shared memory
}

template <int D>
constexpr size_t single_smem() {
    return (size_t)AR_WARPS * SingleStages<D>::value * 2 * AS_KEYS * (D + 8) * 2;
}

int rows_bucket(int d, int dv) {
    const int most = d > dv ? d : dv;
    return most <= 64 ? 64 : (most <= 128 ? 128 : 256);
}

int device_sms() {
    static int sms = 0;
    if (sms <= 0) {
        int dev = 0;
        cudaGetDevice(&dev);
        if (cudaDeviceGetAttribute(&sms, cudaDevAttrMultiProcessorCount, dev) != cudaSuccess || sms <= 0) sms = 148;
    }
    return sms;
}

template <int D, bool POOL>
int launch_rows(const AttentionArgs& p, cudaStream_t s) {
    const int qt = AR_ROWS / (p.nh / p.nkv);
    constexpr int KT = rows_keys<D>();
    constexpr size_t smem = rows_smem<D>();
    int rc = ferris_allow_dynamic_smem((const void*)attention_rows_kernel<D, KT, POOL>, smem);
    if (rc != FERRIS_OK) return rc;
    ferris_launch(attention_rows_kernel<D, KT, POOL>, dim3((p.tokens + qt - 1) / qt, p.nkv), dim3(AR_THREADS), smem, s, p);
    FERRIS_LAUNCH_CHECK();
}

template <int D, bool POOL, bool FAST>
int launch_single_form(const AttentionArgs& p, int splits, cudaStream_t s) {
    const int groups = (p.nh / p.nkv + AS_ROWS - 1) / AS_ROWS;
    constexpr size_t smem = single_smem<D>();
    static_assert((size_t)(AR_WARPS + 1) * AS_ROWS * (D + 2) * sizeof(float) <= smem, "the warps meet in the ring's memory");
    int rc = ferris_allow_dynamic_smem((const void*)attention_single_rows_kernel<D, POOL, FAST>, smem);
    if (rc != FERRIS_OK) return rc;
    const dim3 grid(p.tokens, p.nkv * groups, splits);
    if (splits > 1)
        ferris_launch_cluster(attention_single_rows_kernel<D, POOL, FAST>, grid, dim3(AR_THREADS), smem, s, (unsigned)splits, p, groups, splits);
    else
        ferris_launch(attention_single_rows_kernel<D, POOL, FAST>, grid, dim3(AR_THREADS), smem, s, p, groups, splits);
    FERRIS_LAUNCH_CHECK();
}

template <int D, bool POOL>
int launch_single(const AttentionArgs& p, int splits, cudaStream_t s) {
    const bool fast = !p.values_in_keys && p.d == D && p.dv == D && p.page_size % AS_KEYS == 0;
    return fast ? launch_single_form<D, POOL, true>(p, splits, s) : launch_single_form<D, POOL, false>(p, splits, s);
}

}  // namespace

// Whether ferris_attention_rows takes a geometry (bf16).  portions: 1 = the kernel for portions of prompts, 0 = single tokens.
FERRIS_API int ferris_attention_rows_takes(int nh, int nkv, int d, int dv, int portions) {
    if (nh <= 0 || nkv <= 0 || nh % nkv || d <= 0 || dv <= 0 || d % 8 || dv % 8 || d > 256 || dv > 256) return 0;
    if (nkv > 65535 || (long long)nkv * ((nh / nkv + 7) / 8) > 65535) return 0;
    return portions ? nh / nkv <= AR_ROWS : 1;
}

// Arguments as ferris_paged_attention_simt, bf16 throughout, no distance penalty; v_stride is 0 (values in rows of their own)
// or d, with v_cache the key cache (a value is the first dv elements of its key).  portions:
// requests bring several tokens each (the kernel of 64-row blocks); else kv_span is the most keys a token sees (0: unknown),
// by which they are cut into shares.
FERRIS_API int ferris_attention_rows(const void* q, int ldq, void* out, int ldo, const void* k_cache, const void* v_cache,
                                     const int* block_tables, int max_blocks, const int* token_seq, const int* positions,
                                     int tokens, int nh, int nkv, int d, int dv, int page_size, int window, float scale,
                                     const float* sink, int v_stride, const void* pool_k, const void* pool_v, const int* pool_tables,
                                     int pool_max_blocks, int pool_every, int keep, float softcap, const void* gate, int ldgate,
                                     int portions, int kv_span, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (!ferris_attention_rows_takes(nh, nkv, d, dv, portions))
        FERRIS_REFUSE("attention rows: %d heads over %d kv heads of %d / %d are not taken", nh, nkv, d, dv);
    if (page_size <= 0 || max_blocks <= 0) FERRIS_REFUSE("attention: page_size=%d max_blocks=%d", page_size, max_blocks);
    if (v_stride != 0 && (v_stride != d || dv > d || v_cache != k_cache))
        FERRIS_REFUSE("attention rows: values %d elements apart in keys of %d", v_stride, d);
    const ScoreTerms st = {nullptr, nullptr, nullptr, sink, v_stride, softcap, gate, ldgate};
    const PooledKeys pk = keys_beside(pool_k, pool_v, pool_tables, pool_max_blocks, pool_every, keep, k_cache, v_cache, block_tables, max_blocks);
    if (int rc = check_pooled(pk, window, st)) return rc;
    if ((((uintptr_t)q | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)pool_k | (uintptr_t)pool_v) & 15) != 0 || ldq % 8 ||
        ((uintptr_t)out & 3) || (ldo & 1))
        FERRIS_REFUSE("attention rows: rows must start on 16 bytes");
    const AttentionArgs p = {(const bf16*)q, (bf16*)out, (const bf16*)k_cache, (const bf16*)v_cache, block_tables, token_seq,
                             positions, sink, pk, ldq, ldo, max_blocks, tokens, nh, nkv, d, dv, page_size, window,
                             (softcap > 0.0f ? softcap : scale) * LOG2E, softcap > 0.0f ? scale / softcap : 0.0f,
                             (const bf16*)gate, ldgate, v_stride > 0 ? 1 : 0};
    cudaStream_t s = (cudaStream_t)stream;
    const bool pool = pk.every > 0 || pk.keep > 0;
    const int bucket = rows_bucket(d, dv);
    if (portions) {
        if (bucket == 64) return pool ? launch_rows<64, true>(p, s) : launch_rows<64, false>(p, s);
        if (bucket == 128) return pool ? launch_rows<128, true>(p, s) : launch_rows<128, false>(p, s);
        return pool ? launch_rows<256, true>(p, s) : launch_rows<256, false>(p, s);
    }
    // shares of a token's keys: as many as fill the SMs about twice over (two blocks are resident on one), of 64 keys at least
    int splits = 1;
    if (kv_span > 0) {
        const long long blocks = (long long)tokens * nkv * ((nh / nkv + AS_ROWS - 1) / AS_ROWS);
        long long want = 2LL * device_sms() / blocks;
        if (want > kv_span / 64) want = kv_span / 64;
        if (want > AS_MAX_SPLITS) want = AS_MAX_SPLITS;
        if (want > 1) splits = (int)want;
    }
    if (bucket == 64) return pool ? launch_single<64, true>(p, splits, s) : launch_single<64, false>(p, splits, s);
    if (bucket == 128) return pool ? launch_single<128, true>(p, splits, s) : launch_single<128, false>(p, splits, s);
    return pool ? launch_single<256, true>(p, splits, s) : launch_single<256, false>(p, splits, s);
}
