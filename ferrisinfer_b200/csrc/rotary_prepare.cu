// What stands between the q/k product and attention where queries and keys are normed over their whole projection
// and then rotated, and where the keys as projected may serve as the values:
//
//   q <- q / sqrt(mean(q^2) + eps) * wq      the mean over ALL heads' elements of the token at once (wq spans them)
//   k <- k / sqrt(mean(k^2) + eps) * wk      likewise; either norm is skipped when its weight is null
//   values = the third part of the row, or (values_from_keys) k as projected, before the norm
//   the first R elements of every q and k head rotated by the token's position: the pair (u, v), elements
//   (i, i + R/2) of a head ("half") or (2i, 2i + 1) ("interleaved"), becomes (u c - v s, v c + u s) with
//   c = mag cos(pos * freq[i]), s = mag sin(pos * freq[i]); the other elements pass
//   q rewritten in place, k and the values stored into the paged cache.
//
// Rows: [nh d | nkv d | nkv dv unless values_from_keys].  Everything is computed in fp32 (angles as position_angle
// forms them, sincosf in full precision); one block per token.
//
// Three kernels.  The vector one (no rotation, values of their own): 16 bytes at a time, every element loaded once.  The
// paired one (even head sizes and row strides, rows that start on a pair): a token's cosines and
// sines are formed once in shared memory and serve all its heads, both sums of squares come out of one pass and one
// reduction, and every thread loads, norms, rotates and stores two neighbouring elements at a time (in the
// interleaved layout a pair that rotates together is one such load).  The general one takes every other geometry
// element by element.
//
// Two things may ride along (PrepareExtras).  Value mixing: a layer stores (1 - lambda) v + lambda v1 as its values, v1
// being what another layer projected for the same token in this pass; that layer leaves its rows in a buffer on its
// way.  Pooled blocks: a cache of means, one row for every `pool` consecutive positions; in a step of single tokens the
// block of the token that completes such a run reads the run's keys and values from the pages and writes their mean.
// Steps that bring portions of prompts do the same in a launch of its own behind this one (a run's tokens then lie in
// several blocks of the grid): pool_blocks_kernel.
#include <math.h>
#include <stdint.h>

#include "common.cuh"

namespace {

struct PrepareExtras {
    void* first;            // the rows that values are mixed with, [tokens, nkv * dv] (null: nothing is mixed)
    const float* lambda;    // one number on the device; null: this layer's values are copied INTO `first`
    const int* pool_slots;  // [tokens]: the pooled row that the token completes, or < 0 (null: no pooling here)
    void* pool_k;           // [pages, nkv, page_size, d] and [.., dv]: the pooled rows
    void* pool_v;
    int pool;               // positions to a pooled row
    const int* tables;      // block tables of the unpooled pages, [requests, max_blocks]
    const int* token_seq;
    int max_blocks;
    const float* freq_lo;   // what the 32-bit frequencies lack of their 64-bit values (null: nothing)
};

// Cosine and sine of position x frequency.  With freq_lo the angle keeps the digits that one 32-bit product rounds away: the
// product's own rounding error comes from an FMA, the frequency's from freq_lo, and the small sum e of the two enters as
// sin(a + e) = sin a + e cos a, cos(a + e) = cos a - e sin a.  At position 1,000 a 32-bit angle is off by up to 6e-5 rad, which
// shows in 32-bit logits.
__device__ __forceinline__ void position_angle(float p, const float* __restrict__ freq, const float* __restrict__ freq_lo, int f,
                                               float& s, float& c) {
    const float hi = freq[f], angle = p * hi;
    sincosf(angle, &s, &c);
    if (freq_lo) {
        const float e = fmaf(p, hi, -angle) + p * freq_lo[f];
        const float s0 = s;
        s = fmaf(e, c, s), c = fmaf(-e, s0, c);
    }
}

// The pooled row `slot` = the means of the keys and of the values of positions pos - pool + 1 .. pos, as the pages hold
// them: fp32 sums in the order of the positions, one division, one rounding.  Elements `first`, `first + step`, ... of
// the nkv heads' keys and then of their values.
template <typename T>
__device__ __forceinline__ void pool_run(const T* k_cache, const T* v_cache, const int* table, T* pool_k, T* pool_v, int slot,
                                         int pos, int pool, int nkv, int d, int dv, int page_size, int first, int step) {
    const int nk = nkv * d, total = nk + nkv * dv;
    const int ppage = slot / page_size, pin = slot % page_size;
    for (int e = first; e < total; e += step) {
        const bool key = e < nk;
        const int x = key ? e : e - nk, width = key ? d : dv;
        const int head = x / width, i = x - head * width;
        const T* base = key ? k_cache : v_cache;
        float sum = 0.0f;
        int j = pos - pool + 1;
        while (j <= pos) {  // page by page
            const int in_page = j % page_size;
            const int n = min(page_size - in_page, pos - j + 1);
            const int page = table[j / page_size];
            if (page < 0) return;  // never: a run's pages stay until it is complete
            const T* src = base + (((size_t)page * nkv + head) * page_size + in_page) * width + i;
#pragma unroll 4
            for (int r = 0; r < n; ++r) sum += to_float(src[(size_t)r * width]);
            j += n;
        }
        T* dst = (key ? pool_k : pool_v) + (((size_t)ppage * nkv + head) * page_size + pin) * width + i;
        *dst = from_float<T>(sum / (float)pool);
    }
}

// 16 bytes as fp32 and back: eight bf16 or four floats
template <typename T>
struct Vec16 {
    static constexpr int N = 16 / (int)sizeof(T);
};
__device__ __forceinline__ void widen(const uint4& u, float (&f)[4]) {
    f[0] = __uint_as_float(u.x), f[1] = __uint_as_float(u.y), f[2] = __uint_as_float(u.z), f[3] = __uint_as_float(u.w);
}
__device__ __forceinline__ void widen(const uint4& u, float (&f)[8]) {
    const uint32_t x[4] = {u.x, u.y, u.z, u.w};
#pragma unroll
    for (int i = 0; i < 4; ++i) f[2 * i] = __uint_as_float(x[i] << 16), f[2 * i + 1] = __uint_as_float(x[i] & 0xffff0000u);
}
__device__ __forceinline__ uint4 narrow(const float (&f)[4]) {
    return make_uint4(__float_as_uint(f[0]), __float_as_uint(f[1]), __float_as_uint(f[2]), __float_as_uint(f[3]));
}
__device__ __forceinline__ uint4 narrow(const float (&f)[8]) {
    uint32_t x[4];
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        __nv_bfloat162 v = __floats2bfloat162_rn(f[2 * i], f[2 * i + 1]);
        x[i] = *reinterpret_cast<uint32_t*>(&v);
    }
    return make_uint4(x[0], x[1], x[2], x[3]);
}

// pool_run with 16 bytes of a row at a time (d and dv whole vectors, caches on 16 bytes); every element's sum is formed in
// the same order.
template <typename T>
__device__ __forceinline__ void pool_run_vec(const T* k_cache, const T* v_cache, const int* table, T* pool_k, T* pool_v,
                                             int slot, int pos, int pool, int nkv, int d, int dv, int page_size, int first,
                                             int step) {
    constexpr int E = Vec16<T>::N;
    const int nk = nkv * d / E, total = nk + nkv * dv / E;
    const int ppage = slot / page_size, pin = slot % page_size;
    for (int x = first; x < total; x += step) {
        const bool key = x < nk;
        const int width = key ? d : dv, e = (key ? x : x - nk) * E;
        const int head = e / width, i = e - head * width;
        const T* base = key ? k_cache : v_cache;
        float sum[E];
#pragma unroll
        for (int q = 0; q < E; ++q) sum[q] = 0.0f;
        int j = pos - pool + 1;
        while (j <= pos) {
            const int in_page = j % page_size;
            const int n = min(page_size - in_page, pos - j + 1);
            const int page = table[j / page_size];
            if (page < 0) return;  // never: a run's pages stay until it is complete
            const T* src = base + (((size_t)page * nkv + head) * page_size + in_page) * width + i;
#pragma unroll 8
            for (int r = 0; r < n; ++r) {
                float f[E];
                widen(*reinterpret_cast<const uint4*>(src + (size_t)r * width), f);
#pragma unroll
                for (int q = 0; q < E; ++q) sum[q] += f[q];
            }
            j += n;
        }
#pragma unroll
        for (int q = 0; q < E; ++q) sum[q] /= (float)pool;
        T* dst = (key ? pool_k : pool_v) + (((size_t)ppage * nkv + head) * page_size + pin) * width + i;
        *reinterpret_cast<uint4*>(dst) = narrow(sum);
    }
}

// The pooled rows that the tokens of a step complete, behind the launch that wrote the step's keys and values.
// A block looks at POOL_TOKENS tokens of the step.
constexpr int POOL_TOKENS = 16;
template <typename T, bool VEC>
__global__ void __launch_bounds__(128) pool_blocks_kernel(const T* k_cache, const T* v_cache, T* pool_k, T* pool_v,
                                                          const int* __restrict__ tables, int max_blocks,
                                                          const int* __restrict__ token_seq, const int* __restrict__ positions,
                                                          const int* __restrict__ pool_slots, int tokens, int pool, int nkv,
                                                          int d, int dv, int page_size) {
    pdl_wait();
    pdl_launch_dependents();
    const int t0 = blockIdx.x * POOL_TOKENS, t1 = min(tokens, t0 + POOL_TOKENS);
    for (int t = t0; t < t1; ++t) {
        const int slot = pool_slots[t];
        if (slot < 0) continue;
        const int* table = tables + (size_t)token_seq[t] * max_blocks;
        const int first = blockIdx.y * blockDim.x + threadIdx.x, step = gridDim.y * blockDim.x;
        if (VEC)
            pool_run_vec<T>(k_cache, v_cache, table, pool_k, pool_v, slot, positions[t], pool, nkv, d, dv, page_size, first, step);
        else
            pool_run<T>(k_cache, v_cache, table, pool_k, pool_v, slot, positions[t], pool, nkv, d, dv, page_size, first, step);
    }
}

template <typename T>
__global__ void __launch_bounds__(128) qk_norm_rotary_cache_write_kernel(
    T* qkv, int ld, const int* __restrict__ positions, const int* __restrict__ slot_mapping, T* __restrict__ k_cache,
    T* __restrict__ v_cache, int nh, int nkv, int d, int dv, int page_size, const float* __restrict__ q_weight,
    const float* __restrict__ k_weight, float eps, const float* __restrict__ freq, int rotary, int interleaved, float mag,
    int values_from_keys, int write_kv, const PrepareExtras ex) {
    __shared__ float scratch[33];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int pos = positions[t];
    T* row = qkv + (size_t)t * ld;
    const int nq = nh * d, nk = nkv * d;
    float inv_q = 1.0f, inv_k = 1.0f;
    if (q_weight) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < nq; i += blockDim.x) {
            const float v = to_float(row[i]);
            ss = fmaf(v, v, ss);
        }
        inv_q = 1.0f / sqrtf(block_sum(ss, scratch) / (float)nq + eps);
    }
    if (k_weight) {
        float ss = 0.0f;
        for (int i = threadIdx.x; i < nk; i += blockDim.x) {
            const float v = to_float(row[nq + i]);
            ss = fmaf(v, v, ss);
        }
        inv_k = 1.0f / sqrtf(block_sum(ss, scratch) / (float)nk + eps);
    }
    const int slot = write_kv ? slot_mapping[t] : -1;
    const int page = slot >= 0 ? slot / page_size : 0;
    const int in_page = slot >= 0 ? slot % page_size : 0;
    if (slot >= 0) {  // the values first: where they are the keys as projected, before anything touches those
        const T* vrow = values_from_keys ? row + nq : row + nq + nk;
        T* mixed = reinterpret_cast<T*>(ex.first) + (size_t)t * nkv * dv;
        const float lam = ex.first && ex.lambda ? *ex.lambda : 0.0f;
        for (int e = threadIdx.x; e < nkv * dv; e += blockDim.x) {
            const int h = e / dv, i = e % dv;
            T v = vrow[e];
            if (ex.first) {
                if (ex.lambda)
                    v = from_float<T>(fmaf(lam, to_float(mixed[e]), (1.0f - lam) * to_float(v)));
                else
                    mixed[e] = v;
            }
            v_cache[(((size_t)page * nkv + h) * page_size + in_page) * dv + i] = v;
        }
    }
    const int half = rotary >> 1;
    const int last = slot >= 0 ? nq + nk : nq;  // without a cache to write, the keys are left alone
    for (int e = threadIdx.x; e < last; e += blockDim.x) {
        const bool is_q = e < nq;
        const int h = is_q ? e / d : (e - nq) / d;
        const int i = is_q ? e % d : (e - nq) % d;
        const float inv = is_q ? inv_q : inv_k;
        const float* w = is_q ? q_weight : k_weight;
        const int col = is_q ? e : e - nq;  // the element's place in its projection, where its norm weight lies
        T* dst = is_q ? row + e - i : k_cache + (((size_t)page * nkv + h) * page_size + in_page) * d;
        if (i >= rotary) {
            const float x = to_float(row[e]);
            dst[i] = from_float<T>(w ? (x * inv) * w[col] : x);
            continue;
        }
        // the first member of a pair works for both
        int partner, f;
        if (interleaved) {
            if (i & 1) continue;
            partner = 1, f = i >> 1;
        } else {
            if (i >= half) continue;
            partner = half, f = i;
        }
        float u = to_float(row[e]), v = to_float(row[e + partner]);
        if (w) u = (u * inv) * w[col], v = (v * inv) * w[col + partner];
        float s, c;
        position_angle((float)pos, freq, ex.freq_lo, f, s, c);
        s *= mag, c *= mag;
        dst[i] = from_float<T>(u * c - v * s);
        dst[i + partner] = from_float<T>(v * c + u * s);
    }
    if (ex.pool_slots && slot >= 0 && ex.pool_slots[t] >= 0) {
        __syncthreads();  // the token's own key and value are in their page
        pool_run<T>(k_cache, v_cache, ex.tables + (size_t)ex.token_seq[t] * ex.max_blocks, reinterpret_cast<T*>(ex.pool_k),
                    reinterpret_cast<T*>(ex.pool_v), ex.pool_slots[t], pos, ex.pool, nkv, d, dv, page_size, threadIdx.x, blockDim.x);
    }
}

__device__ __forceinline__ float2 load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load2(const bf16* p) {
    return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p));
}
__device__ __forceinline__ void store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void store2(bf16* p, float a, float b) {
    *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b);
}

// Two sums over a block at once; every thread gets both.  `scratch` holds 66 floats.
__device__ __forceinline__ float2 block_sum2(float a, float b, float* scratch) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    a = warp_sum(a), b = warp_sum(b);
    if (lane == 0) scratch[warp] = a, scratch[32 + warp] = b;
    __syncthreads();
    const int nwarps = (blockDim.x + 31) >> 5;
    if (warp == 0) {
        float x = lane < nwarps ? scratch[lane] : 0.0f, y = lane < nwarps ? scratch[32 + lane] : 0.0f;
        x = warp_sum(x), y = warp_sum(y);
        if (lane == 0) scratch[64] = x, scratch[65] = y;
    }
    __syncthreads();
    return make_float2(scratch[64], scratch[65]);
}

// d, dv, ld, nq, nk even; rows and caches start on a pair of elements.  Dynamic shared memory: `rotary` floats (the
// token's cosines, then its sines, both times mag).
template <typename T, bool INTERLEAVED>
__global__ void __launch_bounds__(256) qk_norm_rotary_cache_write_paired_kernel(
    T* qkv, int ld, const int* __restrict__ positions, const int* __restrict__ slot_mapping, T* __restrict__ k_cache,
    T* __restrict__ v_cache, int nh, int nkv, int d, int dv, int page_size, const float* __restrict__ q_weight,
    const float* __restrict__ k_weight, float eps, const float* __restrict__ freq, int rotary, float mag,
    int values_from_keys, int write_kv, const PrepareExtras ex) {
    extern __shared__ float cs[];
    __shared__ float scratch[66];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int half = rotary >> 1;
    const int pos = positions[t];
    for (int f = threadIdx.x; f < half; f += blockDim.x) {
        float s, c;
        position_angle((float)pos, freq, ex.freq_lo, f, s, c);
        cs[f] = c * mag, cs[half + f] = s * mag;
    }
    const int slot = write_kv ? slot_mapping[t] : -1;
    T* row = qkv + (size_t)t * ld;
    const int nq = nh * d, nk = nkv * d;
    float sq = 0.0f, sk = 0.0f;
    if (q_weight)
        for (int e = 2 * threadIdx.x; e < nq; e += 2 * blockDim.x) {
            const float2 v = load2(row + e);
            sq = fmaf(v.x, v.x, sq), sq = fmaf(v.y, v.y, sq);
        }
    if (k_weight)
        for (int e = 2 * threadIdx.x; e < nk; e += 2 * blockDim.x) {
            const float2 v = load2(row + nq + e);
            sk = fmaf(v.x, v.x, sk), sk = fmaf(v.y, v.y, sk);
        }
    const float2 sums = block_sum2(sq, sk, scratch);  // also: the table is written
    const float inv_q = q_weight ? 1.0f / sqrtf(sums.x / (float)nq + eps) : 1.0f;
    const float inv_k = k_weight ? 1.0f / sqrtf(sums.y / (float)nk + eps) : 1.0f;
    const int page = slot >= 0 ? slot / page_size : 0;
    const int in_page = slot >= 0 ? slot % page_size : 0;
    if (slot >= 0) {
        const T* vrow = values_from_keys ? row + nq : row + nq + nk;
        T* mixed = reinterpret_cast<T*>(ex.first) + (size_t)t * nkv * dv;
        const float lam = ex.first && ex.lambda ? *ex.lambda : 0.0f;
        for (int e = 2 * threadIdx.x; e < nkv * dv; e += 2 * blockDim.x) {
            const int h = e / dv, i = e - h * dv;
            float2 v = load2(vrow + e);
            if (ex.first) {
                if (ex.lambda) {
                    const float2 f = load2(mixed + e);
                    v.x = fmaf(lam, f.x, (1.0f - lam) * v.x), v.y = fmaf(lam, f.y, (1.0f - lam) * v.y);
                } else {
                    store2(mixed + e, v.x, v.y);
                }
            }
            store2(v_cache + (((size_t)page * nkv + h) * page_size + in_page) * dv + i, v.x, v.y);
        }
    }
    const int last = slot >= 0 ? nq + nk : nq;
    const int per_head = d >> 1;  // items of a head: its rotating pairs, then its other elements two by two
    for (int item = threadIdx.x; item < (last >> 1); item += blockDim.x) {
        const int head = item / per_head, j = item - head * per_head;
        const bool is_q = head < nh;
        const int h = is_q ? head : head - nh;
        const float inv = is_q ? inv_q : inv_k;
        const float* w = is_q ? q_weight : k_weight;
        const T* src = row + (size_t)head * d;
        const float* wh = w ? w + (size_t)h * d : nullptr;
        T* dst = is_q ? row + (size_t)head * d : k_cache + (((size_t)page * nkv + h) * page_size + in_page) * d;
        if (j >= half) {  // two elements that pass
            const int i = rotary + 2 * (j - half);
            float2 x = load2(src + i);
            if (w) x.x = (x.x * inv) * wh[i], x.y = (x.y * inv) * wh[i + 1];
            store2(dst + i, x.x, x.y);
            continue;
        }
        const float c = cs[j], s = cs[half + j];
        if (INTERLEAVED) {
            const int i = 2 * j;
            float2 x = load2(src + i);
            if (w) x.x = (x.x * inv) * wh[i], x.y = (x.y * inv) * wh[i + 1];
            store2(dst + i, x.x * c - x.y * s, x.y * c + x.x * s);
        } else {
            float u = to_float(src[j]), v = to_float(src[j + half]);
            if (w) u = (u * inv) * wh[j], v = (v * inv) * wh[j + half];
            dst[j] = from_float<T>(u * c - v * s);
            dst[j + half] = from_float<T>(v * c + u * s);
        }
    }
    if (ex.pool_slots && slot >= 0 && ex.pool_slots[t] >= 0) {
        __syncthreads();  // the token's own key and value are in their page
        pool_run<T>(k_cache, v_cache, ex.tables + (size_t)ex.token_seq[t] * ex.max_blocks, reinterpret_cast<T*>(ex.pool_k),
                    reinterpret_cast<T*>(ex.pool_v), ex.pool_slots[t], pos, ex.pool, nkv, d, dv, page_size, threadIdx.x, blockDim.x);
    }
}

// Without a rotation and with values of their own: rows of whole 16-byte vectors (d, dv, ld multiples of a vector), every
// vector loaded once and kept in registers (VPT a thread) between the sums of squares and the scaling.
template <typename T, int VPT>
__global__ void __launch_bounds__(256) qk_norm_cache_write_vec_kernel(
    T* qkv, int ld, const int* __restrict__ positions, const int* __restrict__ slot_mapping, T* __restrict__ k_cache,
    T* __restrict__ v_cache, int nh, int nkv, int d, int dv, int page_size, const float* __restrict__ q_weight,
    const float* __restrict__ k_weight, float eps, int write_kv, const PrepareExtras ex) {
    constexpr int E = Vec16<T>::N;
    __shared__ float scratch[66];
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int slot = write_kv ? slot_mapping[t] : -1;
    T* row = qkv + (size_t)t * ld;
    const int nq = nh * d, nk = nkv * d, total = (nq + nk + (slot >= 0 ? nkv * dv : 0)) / E;
    const int page = slot >= 0 ? slot / page_size : 0;
    const int in_page = slot >= 0 ? slot % page_size : 0;
    T* mixed = reinterpret_cast<T*>(ex.first) + (size_t)t * nkv * dv;
    uint4 u[VPT], other[VPT];
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int x = threadIdx.x + j * blockDim.x;
        if (x < total) {
            u[j] = *reinterpret_cast<const uint4*>(row + x * E);
            if (ex.first && ex.lambda && x * E >= nq + nk) other[j] = *reinterpret_cast<const uint4*>(mixed + x * E - nq - nk);
        }
    }
    const float lam = ex.first && ex.lambda ? *ex.lambda : 0.0f;
    float sq = 0.0f, sk = 0.0f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int e = (threadIdx.x + j * blockDim.x) * E;
        if (e < nq + nk) {
            float f[E];
            widen(u[j], f);
            float ss = 0.0f;
#pragma unroll
            for (int i = 0; i < E; ++i) ss = fmaf(f[i], f[i], ss);
            if (e < nq) sq += ss; else sk += ss;
        }
    }
    const float2 sums = block_sum2(sq, sk, scratch);
    const float inv_q = q_weight ? 1.0f / sqrtf(sums.x / (float)nq + eps) : 1.0f;
    const float inv_k = k_weight ? 1.0f / sqrtf(sums.y / (float)nk + eps) : 1.0f;
#pragma unroll
    for (int j = 0; j < VPT; ++j) {
        const int x = threadIdx.x + j * blockDim.x, e = x * E;
        if (x >= total) continue;
        float f[E];
        widen(u[j], f);
        if (e < nq + nk) {  // without a cache to write, the keys are left alone
            const bool is_q = e < nq;
            if (!is_q && slot < 0) continue;
            const int col = is_q ? e : e - nq;
            const float* w = is_q ? q_weight : k_weight;
            const float inv = is_q ? inv_q : inv_k;
            if (w) {
#pragma unroll
                for (int i = 0; i < E; i += 4) {
                    const float4 g = *reinterpret_cast<const float4*>(w + col + i);
                    f[i] = (f[i] * inv) * g.x, f[i + 1] = (f[i + 1] * inv) * g.y;
                    f[i + 2] = (f[i + 2] * inv) * g.z, f[i + 3] = (f[i + 3] * inv) * g.w;
                }
            }
            const int head = col / d;
            T* dst = is_q ? row + e : k_cache + (((size_t)page * nkv + head) * page_size + in_page) * d + col - head * d;
            *reinterpret_cast<uint4*>(dst) = narrow(f);
            continue;
        }
        const int col = e - nq - nk, head = col / dv;
        if (ex.first) {
            if (ex.lambda) {
                float o[E];
                widen(other[j], o);
#pragma unroll
                for (int i = 0; i < E; ++i) f[i] = fmaf(lam, o[i], (1.0f - lam) * f[i]);
            } else {
                *reinterpret_cast<uint4*>(mixed + col) = u[j];
            }
        }
        *reinterpret_cast<uint4*>(v_cache + (((size_t)page * nkv + head) * page_size + in_page) * dv + col - head * dv) = narrow(f);
    }
    if (ex.pool_slots && slot >= 0 && ex.pool_slots[t] >= 0) {
        __syncthreads();  // the token's own key and value are in their page
        pool_run_vec<T>(k_cache, v_cache, ex.tables + (size_t)ex.token_seq[t] * ex.max_blocks, reinterpret_cast<T*>(ex.pool_k),
                        reinterpret_cast<T*>(ex.pool_v), ex.pool_slots[t], positions[t], ex.pool, nkv, d, dv, page_size,
                        threadIdx.x, blockDim.x);
    }
}

// The norm per HEAD: every q and k head divided by the root mean square of its own d elements and multiplied by a
// weight of d numbers that all heads share (wq for queries, wk for keys; null: that side is not normed), then rotated
// and stored as above.  A warp per head: its lanes sum the head's squares, then norm, rotate and store it; the values
// are copied by the whole block.
template <typename T>
__global__ void __launch_bounds__(256) qk_head_norm_rotary_cache_write_kernel(
    T* qkv, int ld, const int* __restrict__ positions, const int* __restrict__ slot_mapping, T* __restrict__ k_cache,
    T* __restrict__ v_cache, int nh, int nkv, int d, int dv, int page_size, const float* __restrict__ q_weight,
    const float* __restrict__ k_weight, float eps, const float* __restrict__ freq, int rotary, int interleaved, float mag,
    int write_kv, const float* __restrict__ freq_lo) {
    extern __shared__ float cs[];  // the token's cosines, then its sines, both times mag
    pdl_wait();
    pdl_launch_dependents();
    const int t = blockIdx.x;
    const int pos = positions[t];
    const int half = rotary >> 1;
    for (int f = threadIdx.x; f < half; f += blockDim.x) {
        float s, c;
        position_angle((float)pos, freq, freq_lo, f, s, c);
        cs[f] = c * mag, cs[half + f] = s * mag;
    }
    __syncthreads();
    T* row = qkv + (size_t)t * ld;
    const int nq = nh * d, nk = nkv * d;
    const int slot = write_kv ? slot_mapping[t] : -1;
    const int page = slot >= 0 ? slot / page_size : 0;
    const int in_page = slot >= 0 ? slot % page_size : 0;
    if (slot >= 0) {
        const T* vrow = row + nq + nk;
        for (int e = threadIdx.x; e < nkv * dv; e += blockDim.x) {
            const int h = e / dv, i = e - h * dv;
            v_cache[(((size_t)page * nkv + h) * page_size + in_page) * dv + i] = vrow[e];
        }
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    const int heads = slot >= 0 ? nh + nkv : nh;  // without a cache to write, the keys are left alone
    for (int head = warp; head < heads; head += warps) {
        const bool is_q = head < nh;
        const int h = is_q ? head : head - nh;
        const float* w = is_q ? q_weight : k_weight;
        const T* src = row + (size_t)head * d;
        T* dst = is_q ? row + (size_t)head * d : k_cache + (((size_t)page * nkv + h) * page_size + in_page) * d;
        float inv = 1.0f;
        if (w) {
            float ss = 0.0f;
            for (int i = lane; i < d; i += 32) {
                const float x = to_float(src[i]);
                ss = fmaf(x, x, ss);
            }
            inv = 1.0f / sqrtf(warp_sum(ss) / (float)d + eps);  // every lane has read the head before any lane writes it
        }
        for (int j = lane; j < half; j += 32) {
            const int i0 = interleaved ? 2 * j : j, i1 = interleaved ? 2 * j + 1 : j + half;
            float u = to_float(src[i0]), v = to_float(src[i1]);
            if (w) u = (u * inv) * w[i0], v = (v * inv) * w[i1];
            const float c = cs[j], s = cs[half + j];
            dst[i0] = from_float<T>(u * c - v * s);
            dst[i1] = from_float<T>(v * c + u * s);
        }
        for (int i = rotary + lane; i < d; i += 32) {
            const float x = to_float(src[i]);
            dst[i] = from_float<T>(w ? (x * inv) * w[i] : x);
        }
    }
}

}  // namespace

FERRIS_API int ferris_qk_norm_rotary_cache_write(void* qkv, int ld, int dtype, const int* positions,
                                                 const int* slot_mapping, void* k_cache, void* v_cache, int tokens, int nh,
                                                 int nkv, int d, int dv, int page_size, const float* q_weight,
                                                 const float* k_weight, float eps, const float* freq, int rotary,
                                                 int interleaved, float mag, int values_from_keys, int write_kv,
                                                 void* first_values, const float* mix_lambda, const int* pool_slots,
                                                 void* pool_k, void* pool_v, int pool, const int* tables, int max_blocks,
                                                 const int* token_seq, const float* freq_lo, void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (mix_lambda && !first_values) FERRIS_REFUSE("qk norm + rotation: nothing to mix the values with");
    if (first_values && !write_kv) FERRIS_REFUSE("qk norm + rotation: values are mixed where they are stored");
    if (pool_slots && (!write_kv || !pool_k || !pool_v || pool <= 0 || !tables || max_blocks <= 0 || !token_seq))
        FERRIS_REFUSE("qk norm + rotation: pooled rows of %d positions want a cache, pooled pages and block tables", pool);
    const PrepareExtras ex = {first_values, mix_lambda, pool_slots, pool_k, pool_v, pool, tables, token_seq, max_blocks, freq_lo};
    if (nh <= 0 || nkv <= 0 || d <= 0 || dv <= 0 || page_size <= 0)
        FERRIS_REFUSE("qk norm + rotation: nh=%d nkv=%d d=%d dv=%d page_size=%d", nh, nkv, d, dv, page_size);
    if (rotary < 0 || rotary > d || (rotary & 1) || (rotary > 0 && !freq))
        FERRIS_REFUSE("qk norm + rotation: %d rotated elements of heads of %d", rotary, d);
    if (values_from_keys && dv != d) FERRIS_REFUSE("qk norm + rotation: keys of %d cannot serve as values of %d", d, dv);
    if (ld < (nh + nkv) * d + (values_from_keys ? 0 : nkv * dv)) FERRIS_REFUSE("qk norm + rotation: rows of %d are too short", ld);
    if (write_kv && (!slot_mapping || !k_cache || !v_cache)) FERRIS_REFUSE("qk norm + rotation: no cache to write");
    cudaStream_t s = (cudaStream_t)stream;
    const size_t elem = dtype == FERRIS_F32 ? 4 : 2;
    const int E = (int)(16 / elem);
    const long long vectors = ((long long)(nh + nkv) * d + (long long)nkv * dv) / E;
    if (rotary == 0 && !values_from_keys && (dtype == FERRIS_F32 || dtype == FERRIS_BF16) && d % E == 0 && dv % E == 0 && ld % E == 0 &&
        vectors <= 4 * 256 && (((uintptr_t)qkv | (uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)first_values | (uintptr_t)pool_k |
        (uintptr_t)pool_v | (uintptr_t)q_weight | (uintptr_t)k_weight) & 15) == 0) {
        const dim3 block(vectors < 256 ? (unsigned)((vectors + 31) / 32 * 32) : 256);
#define FERRIS_QK_VEC(T, VPT)                                                                                              \
    ferris_launch(qk_norm_cache_write_vec_kernel<T, VPT>, dim3(tokens), block, 0, s, (T*)qkv, ld, positions, slot_mapping,  \
                  (T*)k_cache, (T*)v_cache, nh, nkv, d, dv, page_size, q_weight, k_weight, eps, write_kv, ex)
        const int vpt = (int)((vectors + 255) / 256);
        if (dtype == FERRIS_F32) {
            if (vpt <= 1) FERRIS_QK_VEC(float, 1); else if (vpt <= 2) FERRIS_QK_VEC(float, 2); else FERRIS_QK_VEC(float, 4);
        } else {
            if (vpt <= 1) FERRIS_QK_VEC(bf16, 1); else if (vpt <= 2) FERRIS_QK_VEC(bf16, 2); else FERRIS_QK_VEC(bf16, 4);
        }
#undef FERRIS_QK_VEC
        FERRIS_LAUNCH_CHECK();
    }
    const bool paired = !((d | dv | ld) & 1) && (uintptr_t)qkv % (2 * elem) == 0 && (uintptr_t)k_cache % (2 * elem) == 0 &&
                        (uintptr_t)v_cache % (2 * elem) == 0 && (uintptr_t)first_values % (2 * elem) == 0 && ((uintptr_t)q_weight | (uintptr_t)k_weight) % 8 == 0 &&
                        (dtype == FERRIS_F32 || dtype == FERRIS_BF16);
    if (paired) {
        const size_t smem = (size_t)rotary * sizeof(float);
#define FERRIS_PAIRED(T, I)                                                                                              \
    ferris_launch(qk_norm_rotary_cache_write_paired_kernel<T, I>, dim3(tokens), dim3(256), smem, s, (T*)qkv, ld, positions, \
                  slot_mapping, (T*)k_cache, (T*)v_cache, nh, nkv, d, dv, page_size, q_weight, k_weight, eps, freq, rotary,  \
                  mag, values_from_keys, write_kv, ex)
        if (dtype == FERRIS_F32) {
            if (interleaved) FERRIS_PAIRED(float, true); else FERRIS_PAIRED(float, false);
        } else {
            if (interleaved) FERRIS_PAIRED(bf16, true); else FERRIS_PAIRED(bf16, false);
        }
#undef FERRIS_PAIRED
        FERRIS_LAUNCH_CHECK();
    }
    if (dtype == FERRIS_F32)
        ferris_launch(qk_norm_rotary_cache_write_kernel<float>, dim3(tokens), dim3(128), 0, s, (float*)qkv, ld, positions,
                      slot_mapping, (float*)k_cache, (float*)v_cache, nh, nkv, d, dv, page_size, q_weight, k_weight, eps,
                      freq, rotary, interleaved, mag, values_from_keys, write_kv, ex);
    else if (dtype == FERRIS_BF16)
        ferris_launch(qk_norm_rotary_cache_write_kernel<bf16>, dim3(tokens), dim3(128), 0, s, (bf16*)qkv, ld, positions,
                      slot_mapping, (bf16*)k_cache, (bf16*)v_cache, nh, nkv, d, dv, page_size, q_weight, k_weight, eps,
                      freq, rotary, interleaved, mag, values_from_keys, write_kv, ex);
    else
        FERRIS_REFUSE("qk norm + rotation: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}

// As above with the norm taken per head: q_weight, k_weight fp32 [d] (shared by the heads; null: no norm on that side).
// freq_lo (may be null): fp32 [rotary / 2], the 64-bit frequencies minus their 32-bit roundings.
FERRIS_API int ferris_qk_head_norm_rotary_cache_write(void* qkv, int ld, int dtype, const int* positions,
                                                      const int* slot_mapping, void* k_cache, void* v_cache, int tokens,
                                                      int nh, int nkv, int d, int dv, int page_size, const float* q_weight,
                                                      const float* k_weight, float eps, const float* freq, int rotary,
                                                      int interleaved, float mag, int write_kv, const float* freq_lo,
                                                      void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (nh <= 0 || nkv <= 0 || d <= 0 || dv <= 0 || page_size <= 0)
        FERRIS_REFUSE("head norm + rotation: nh=%d nkv=%d d=%d dv=%d page_size=%d", nh, nkv, d, dv, page_size);
    if (rotary < 0 || rotary > d || (rotary & 1) || (rotary > 0 && !freq))
        FERRIS_REFUSE("head norm + rotation: %d rotated elements of heads of %d", rotary, d);
    if (ld < (nh + nkv) * d + nkv * dv) FERRIS_REFUSE("head norm + rotation: rows of %d are too short", ld);
    if (write_kv && (!slot_mapping || !k_cache || !v_cache)) FERRIS_REFUSE("head norm + rotation: no cache to write");
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = (size_t)(rotary > 0 ? rotary : 1) * sizeof(float);
    const int threads = (nh + nkv) >= 8 ? 256 : 128;
    if (dtype == FERRIS_F32)
        ferris_launch(qk_head_norm_rotary_cache_write_kernel<float>, dim3(tokens), dim3(threads), smem, s, (float*)qkv, ld,
                      positions, slot_mapping, (float*)k_cache, (float*)v_cache, nh, nkv, d, dv, page_size, q_weight, k_weight,
                      eps, freq, rotary, interleaved, mag, write_kv, freq_lo);
    else if (dtype == FERRIS_BF16)
        ferris_launch(qk_head_norm_rotary_cache_write_kernel<bf16>, dim3(tokens), dim3(threads), smem, s, (bf16*)qkv, ld,
                      positions, slot_mapping, (bf16*)k_cache, (bf16*)v_cache, nh, nkv, d, dv, page_size, q_weight, k_weight, eps,
                      freq, rotary, interleaved, mag, write_kv, freq_lo);
    else
        FERRIS_REFUSE("head norm + rotation: unknown dtype %d", dtype);
    FERRIS_LAUNCH_CHECK();
}

// Pooled rows of the tokens of a step whose slot in `pool_slots` is not negative: the means of the `pool` keys and values up
// to the token's position, read from the pages that `tables` [requests, max_blocks] name.
FERRIS_API int ferris_pool_blocks(const void* k_cache, const void* v_cache, void* pool_k, void* pool_v, int dtype,
                                  const int* tables, int max_blocks, const int* token_seq, const int* positions,
                                  const int* pool_slots, int tokens, int pool, int nkv, int d, int dv, int page_size,
                                  void* stream) {
    if (tokens <= 0) return FERRIS_OK;
    if (pool <= 0 || nkv <= 0 || d <= 0 || dv <= 0 || page_size <= 0 || max_blocks <= 0)
        FERRIS_REFUSE("pooled rows: pool=%d nkv=%d d=%d dv=%d page_size=%d max_blocks=%d", pool, nkv, d, dv, page_size, max_blocks);
    if (dtype != FERRIS_F32 && dtype != FERRIS_BF16) FERRIS_REFUSE("pooled rows: unknown dtype %d", dtype);
    const int E = dtype == FERRIS_F32 ? 4 : 8;
    const bool vec = d % E == 0 && dv % E == 0 &&
                     (((uintptr_t)k_cache | (uintptr_t)v_cache | (uintptr_t)pool_k | (uintptr_t)pool_v) & 15) == 0;
    const int items = vec ? nkv * (d + dv) / E : nkv * (d + dv), slabs = (items + 127) / 128;
    const dim3 grid((tokens + POOL_TOKENS - 1) / POOL_TOKENS, slabs < 64 ? slabs : 64), block(128);
    cudaStream_t s = (cudaStream_t)stream;
#define FERRIS_POOL(T, VEC)                                                                                                \
    ferris_launch(pool_blocks_kernel<T, VEC>, grid, block, 0, s, (const T*)k_cache, (const T*)v_cache, (T*)pool_k, (T*)pool_v, \
                  tables, max_blocks, token_seq, positions, pool_slots, tokens, pool, nkv, d, dv, page_size)
    if (dtype == FERRIS_F32) {
        if (vec) FERRIS_POOL(float, true); else FERRIS_POOL(float, false);
    } else {
        if (vec) FERRIS_POOL(bf16, true); else FERRIS_POOL(bf16, false);
    }
#undef FERRIS_POOL
    FERRIS_LAUNCH_CHECK();
}
