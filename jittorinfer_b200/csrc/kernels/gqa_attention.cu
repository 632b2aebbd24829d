// Grouped-query attention over paged key / value rows: H query heads share G key / value heads (head h reads h / (H / G)).
// A cached row holds the normed and rotated keys of a token (G * D columns), then its values (G * V columns).
//
//   gqa_qkv_post    per-head RMS norm of q and k (or none; with weights ahead of the rotation, without after it), RoPE on the first rot
//                   dimensions, a blend of the values with another layer's, rows into the cache
//   gqa_pool        means of the cached rows of complete blocks of positions (single tokens: part of gqa_qkv_post)
//   gqa_attention   scores * scale, softcap, causal mask with a sliding window and / or chunks counted from position 0, one more key per
//                   block of positions that has left the window, softmax with or without a sink (a key without a value, of score 0 or of a
//                   number per head), a gate per head or channel: any mix of portions and single
//                   tokens, keys split over a thread-block cluster.  bf16 heads whose sizes are multiples of 16: products on the
//                   tensor cores (gqa_mma); fp32 and other sizes: CUDA cores (gqa_attention).  Prompts with heads of 128 have a
//                   kernel of their own (mha_prefill_tcgen05.cu).
//
// Activations and cache rows bf16 or fp32; norms, angles, scores and softmax fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "gqa_mask.cuh"
#include "jib_kernels.h"
#include "pdl.cuh"
#include "sm100.cuh"

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ void put(bf16 * p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void put(float * p, float v) { *p = v; }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
template <typename T> __device__ __forceinline__ float exp_t(float v);
template <> __device__ __forceinline__ float exp_t<bf16>(float v) { return __expf(v); }
template <> __device__ __forceinline__ float exp_t<float>(float v) { return expf(v); }
template <typename T> __device__ __forceinline__ float capped(float s, float cap);
template <> __device__ __forceinline__ float capped<bf16>(float s, float cap) {
    return cap * (1.f - __fdividef(2.f, 1.f + __expf(2.f * fminf(s / cap, 40.f))));         // tanh, absolute error ~ 1e-7
}
template <> __device__ __forceinline__ float capped<float>(float s, float cap) { return cap * tanhf(s / cap); }

// 4 adjacent elements of aligned rows, kept as stored until they are needed
template <typename T> struct Vec4;
template <> struct Vec4<float> {
    float4 r;
    __device__ __forceinline__ void load(const float * p) { r = *(const float4 *) p; }
    __device__ __forceinline__ float4 get() const { return r; }
    static __device__ __forceinline__ void store(float * p, float4 v) { *(float4 *) p = v; }
};
template <> struct Vec4<bf16> {
    uint2 r;
    __device__ __forceinline__ void load(const bf16 * p) { r = *(const uint2 *) p; }
    __device__ __forceinline__ float4 get() const {
        const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *) &r.x), y = __bfloat1622float2(*(const __nv_bfloat162 *) &r.y);
        return make_float4(x.x, x.y, y.x, y.y);
    }
    static __device__ __forceinline__ void store(bf16 * p, float4 v) {
        uint2 x;
        *(__nv_bfloat162 *) &x.x = __floats2bfloat162_rn(v.x, v.y);
        *(__nv_bfloat162 *) &x.y = __floats2bfloat162_rn(v.z, v.w);
        *(uint2 *) p = x;
    }
};

// The pooled block a CTA of a portion works on: one CTA (blockIdx.x) per block that can end in this batch.  Sequence b's begin at index
// q_start[b] / pool_size + b, the first is the one its first new position lies in; indices in the gaps have none.
__device__ __forceinline__ bool pool_block(const jib_gqa & a, int & b, int & block) {
    const int P = a.pool_size;
    int hi = a.n_seqs;
    b = 0;
    while (hi - b > 1) {
        const int mid = (b + hi) >> 1;
        if (a.q_start[mid] / P + mid <= (int) blockIdx.x) b = mid; else hi = mid;
    }
    const int q0 = a.q_start[b], n = a.q_start[b + 1] - q0, S = a.seq_lens[b];
    if (n <= 0 || S < n) return false;
    block = (S - n) / P + (int) blockIdx.x - (q0 / P + b);
    return block >= (S - n) / P && (block + 1) * P <= S;
}

// ---- norm, rotation, cache rows: one warp per (token, head of q / k / v) ------------------------------------------------------
constexpr int POST_D = 16;                                   // elements of a head per lane (N): D <= 32 * POST_D

template <typename T, int N>
__global__ void __launch_bounds__(256) gqa_qkv_post_kernel(const __grid_constant__ jib_gqa a, const T * __restrict__ q, const T * __restrict__ k,
                                                           const T * __restrict__ v, long long ld, const float * __restrict__ q_norm,
                                                           const float * __restrict__ k_norm, const float * __restrict__ rope,
                                                           const int * __restrict__ slot_mapping, T * __restrict__ q_out, int single) {
    extern __shared__ float heads[];                         // [8 warps][D]
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, t = blockIdx.y, item = blockIdx.x * 8 + warp;
    const int D = a.D, V = a.V, H = a.H, G = a.G;
    if (item >= H + 2 * G) return;
    T * row = nullptr;
    if (item >= H) {
        const long long slot = slot_mapping[t];
        if (slot >= a.n_slots) {
            if (lane == 0) jib_report(a.status, JIB_ERR_BOUNDS, 48, (int) slot);
            return;
        }
        if (slot < 0) return;                                // a padding row
        row = (T *) a.cache + (size_t) slot * a.row;
    }
    // single tokens: one that completes a block of positions also stores the mean of its rows (the others' are in the cache)
    const int * bt = nullptr;
    T * pooled = nullptr;
    int pos = a.positions[t];
    if (row != nullptr && single && a.pool_size > 0 && pos >= 0 && (pos + 1) % a.pool_size == 0) {
        bt = a.block_tables + (size_t) t * a.max_blocks;
        pooled = (T *) a.pool + gqa_pool_row(bt, pos / a.pool_size, a.pool_size, a.pool_rows, a.block_size) * a.row;
    }
    auto earlier = [&](int col) {                            // sum over the block's earlier rows
        float s = 0.f;
#pragma unroll 4
        for (int p = pos - a.pool_size + 1; p < pos; ++p)
            s += to_f(((const T *) a.cache)[((long long) bt[p / a.block_size] * a.block_size + p % a.block_size) * a.row + col]);
        return s;
    };
    if (item >= H + G) {
        const int g = item - H - G;
        const T * src = v + (size_t) t * ld + g * V, * first = (const T *) a.v_first + (size_t) t * a.ld_first + g * V;
        T * dst = row + G * D + g * V;
        for (int c = lane; c < V; c += 32) {
            T y = src[c];
            if (a.mix_v) put(&y, (1.f - a.v_mix) * to_f(y) + a.v_mix * to_f(first[c]));
            dst[c] = y;
            if (pooled != nullptr) put(pooled + G * D + g * V + c, (earlier(G * D + g * V + c) + to_f(y)) / (float) a.pool_size);
        }
        return;
    }
    const bool is_q = item < H;
    const int head = is_q ? item : item - H;
    const T * src = (is_q ? q : k) + (size_t) t * ld + head * D;
    const float * w = is_q ? q_norm : k_norm;
    float * x = heads + warp * D;
    float e[N], ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = lane + 32 * i;
        e[i] = c < D ? to_f(src[c]) : 0.f;
        ss += e[i] * e[i];
    }
    int at = pos;
    if (at < 0 || at >= a.max_pos) {
        if (lane == 0) jib_report(a.status, JIB_ERR_BOUNDS, 49, at);
        at = 0;
    }
    const int half = a.rot / 2;
    const float2 * cs = (const float2 *) rope + (size_t) at * half;
    float wt[N];
    float2 r[N];
#pragma unroll
    for (int i = 0; i < N; ++i) {                            // requested before the reduction
        const int c = lane + 32 * i;
        wt[i] = w != nullptr && c < D ? w[c] : 0.f;
        r[i] = c < a.rot ? cs[a.neighbours ? c >> 1 : c < half ? c : c - half] : make_float2(1.f, 0.f);
    }
    if (w != nullptr) {
        const float inv = rsqrtf(warp_sum(ss) / (float) D + a.eps);
#pragma unroll
        for (int i = 0; i < N; ++i) e[i] *= inv * wt[i];
    }
#pragma unroll
    for (int i = 0; i < N; ++i)
        if (lane + 32 * i < D) x[lane + 32 * i] = e[i];
    __syncwarp();
    T * dst = is_q ? q_out + ((size_t) t * H + head) * D : row + head * D;
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = lane + 32 * i;
        if (c >= D) continue;
        if (a.neighbours) {
            if (c < a.rot) e[i] = e[i] * r[i].x + ((c & 1) ? x[c - 1] : -x[c + 1]) * r[i].y;
        } else if (c < half) {
            e[i] = e[i] * r[i].x - x[c + half] * r[i].y;
        } else if (c < a.rot) {
            e[i] = e[i] * r[i].x + x[c - half] * r[i].y;
        }
        ss += e[i] * e[i];
    }
    const float inv = a.unit ? rsqrtf(warp_sum(ss) / (float) D + a.eps) : 1.f;
#pragma unroll
    for (int i = 0; i < N; ++i) {
        const int c = lane + 32 * i;
        if (c >= D) continue;
        T y;
        put(&y, e[i] * inv);
        dst[c] = y;
        if (pooled != nullptr) put(pooled + head * D + c, (earlier(head * D + c) + to_f(y)) / (float) a.pool_size);
    }
}

// The same for rotated neighbours (and no norm weights) where whole vectors of 4 can be read: a lane holds 4 adjacent elements, two pairs, and
// the warp takes TOK tokens at a time.  D, V <= 128 * N.
template <typename T, int N, int TOK>
__global__ void __launch_bounds__(256) gqa_pairs_post_kernel(const __grid_constant__ jib_gqa a, const T * __restrict__ q, const T * __restrict__ k,
                                                             const T * __restrict__ v, long long ld, const float * __restrict__ rope,
                                                             const int * __restrict__ slot_mapping, T * __restrict__ q_out) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int lane = threadIdx.x & 31, item = blockIdx.x * 8 + (threadIdx.x >> 5), t0 = blockIdx.y * TOK;
    const int D = a.D, V = a.V, H = a.H, G = a.G;
    if (item >= H + 2 * G) return;
    const bool is_q = item < H, is_v = item >= H + G;
    const int head = is_q ? item : is_v ? item - H - G : item - H, n = is_v ? V : D;
    Vec4<T> x[TOK][N], y[TOK][N];
    T * dst[TOK];
    float4 cs[TOK][N];                                       // cos, sin of the two pairs
#pragma unroll
    for (int j = 0; j < TOK; ++j) {                          // everything is requested before any of it is used
        const int t = min(t0 + j, a.T - 1);
        dst[j] = nullptr;
        if (t0 + j < a.T) {
            if (is_q) {
                dst[j] = q_out + ((size_t) t * H + head) * D;
            } else {
                const long long slot = slot_mapping[t];
                if (slot >= a.n_slots) {
                    if (lane == 0) jib_report(a.status, JIB_ERR_BOUNDS, 48, (int) slot);
                } else if (slot >= 0) {
                    dst[j] = (T *) a.cache + (size_t) slot * a.row + (is_v ? G * D : 0) + head * n;
                }
            }
        }
        int at = a.positions[t];
        if (!is_v && (at < 0 || at >= a.max_pos)) {
            if (lane == 0) jib_report(a.status, JIB_ERR_BOUNDS, 49, at);
            at = 0;
        }
        const T * src = (is_q ? q : is_v ? v : k) + (size_t) t * ld + head * n, * first = (const T *) a.v_first + (size_t) t * a.ld_first + head * n;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const int c = 4 * (lane + 32 * i);
            if (c >= n) continue;
            x[j][i].load(src + c);
            if (is_v && a.mix_v) y[j][i].load(first + c);
            cs[j][i] = make_float4(1.f, 0.f, 1.f, 0.f);
            if (!is_v && c < a.rot) {
                const float2 * r = (const float2 *) rope + (size_t) at * (a.rot / 2) + c / 2;
                const float2 r0 = r[0], r1 = c + 2 < a.rot ? r[1] : make_float2(1.f, 0.f);
                cs[j][i] = make_float4(r0.x, r0.y, r1.x, r1.y);
            }
        }
    }
#pragma unroll
    for (int j = 0; j < TOK; ++j) {
        float4 e[N];
        float ss = 0.f;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            if (4 * (lane + 32 * i) >= n) continue;
            const float4 z = x[j][i].get(), r = cs[j][i];
            if (is_v) {
                e[i] = z;
                if (a.mix_v) {
                    const float4 w = y[j][i].get();
                    const float m = a.v_mix, o = 1.f - m;
                    e[i] = make_float4(o * z.x + m * w.x, o * z.y + m * w.y, o * z.z + m * w.z, o * z.w + m * w.w);
                }
            } else {
                e[i] = make_float4(z.x * r.x - z.y * r.y, z.y * r.x + z.x * r.y, z.z * r.z - z.w * r.w, z.w * r.z + z.z * r.w);
                ss += e[i].x * e[i].x + e[i].y * e[i].y + e[i].z * e[i].z + e[i].w * e[i].w;
            }
        }
        const float inv = a.unit && !is_v ? rsqrtf(warp_sum(ss) / (float) D + a.eps) : 1.f;
        if (dst[j] == nullptr) continue;
#pragma unroll
        for (int i = 0; i < N; ++i) {
            const int c = 4 * (lane + 32 * i);
            if (c < n) Vec4<T>::store(dst[j] + c, make_float4(e[i].x * inv, e[i].y * inv, e[i].z * inv, e[i].w * inv));
        }
    }
}

// Means of complete blocks of pool_size positions, portions, where whole 16-byte vectors can be read: see gqa_pool_kernel; blockIdx.y takes 32
// vectors of the row, 8 threads share one's rows.
template <typename T>
__global__ void __launch_bounds__(256) gqa_pool_vec_kernel(const __grid_constant__ jib_gqa a) {
    constexpr int E = 16 / sizeof(T);
    __shared__ float part[8][32][E + 1];
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int b, block;
    if (!pool_block(a, b, block)) return;
    const int P = a.pool_size, lane = threadIdx.x & 31, g = threadIdx.x >> 5, c = (blockIdx.y * 32 + lane) * E;
    const bool in = c < a.G * (a.D + a.V);
    const int * bt = a.block_tables + (size_t) b * a.max_blocks;
    float s[E];
#pragma unroll
    for (int e = 0; e < E; ++e) s[e] = 0.f;
    if (in) {
#pragma unroll 4
        for (int p = block * P + g; p < block * P + P; p += 8) {
            const uint4 r = *(const uint4 *) ((const T *) a.cache + ((long long) bt[p / a.block_size] * a.block_size + p % a.block_size) * a.row + c);
#pragma unroll
            for (int e = 0; e < E; ++e) s[e] += to_f(((const T *) &r)[e]);
        }
    }
#pragma unroll
    for (int e = 0; e < E; ++e) part[g][lane][e] = s[e];
    __syncthreads();
    if (g > 0 || !in) return;
    T out[E];
#pragma unroll
    for (int e = 0; e < E; ++e) {
        float x = 0.f;
#pragma unroll
        for (int k = 0; k < 8; ++k) x += part[k][lane][e];
        put(out + e, x / (float) P);
    }
    T * dst = (T *) a.pool + gqa_pool_row(bt, block, P, a.pool_rows, a.block_size) * a.row + c;
    uint4 r;
    memcpy(&r, out, 16);
    *(uint4 *) dst = r;
}

// Any sizes.
template <typename T>
__global__ void __launch_bounds__(256) gqa_pool_kernel(const __grid_constant__ jib_gqa a) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int b, block;
    if (!pool_block(a, b, block)) return;
    const int P = a.pool_size, p0 = block * P;
    const int * bt = a.block_tables + (size_t) b * a.max_blocks;
    T * dst = (T *) a.pool + gqa_pool_row(bt, block, P, a.pool_rows, a.block_size) * a.row;
    const int cols = a.G * (a.D + a.V);
    for (int c = threadIdx.x; c < cols; c += 256) {
        float s = 0.f;
#pragma unroll 8
        for (int p = p0; p < p0 + P; ++p) s += to_f(((const T *) a.cache)[((long long) bt[p / a.block_size] * a.block_size + p % a.block_size) * a.row + c]);
        put(dst + c, s / (float) P);
    }
}

// ---- attention on CUDA cores ---------------------------------------------------------------------------------------------------
// A CTA takes up to 16 (token, head) rows that share a key / value head: a run of tokens of one sequence x a run of the head's
// queries.  Key tiles of KT rows are staged in fp32; the tiles the run can see are dealt to the CTAs of a cluster (blockIdx.z), whose
// partial results meet in distributed shared memory.
constexpr int ROWS = 16, NT = 128;

__device__ __forceinline__ void cluster_sync() { asm volatile("barrier.cluster.arrive.release;\n\tbarrier.cluster.wait.acquire;" ::: "memory"); }
__device__ __forceinline__ float ld_peer(const float * p, int rank) {
    uint32_t remote;
    float v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"((uint32_t) __cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("ld.shared::cluster.f32 %0, [%1];" : "=f"(v) : "r"(remote) : "memory");
    return v;
}

// 4 elements c .. c + 3 of a row of n, zero past its end; kept as stored until they are needed (many loads in flight)
template <typename T> struct Quad;
template <> struct Quad<float> {
    float4 r;
    __device__ __forceinline__ void zero() { r = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void load(const float * p, int c, int n, bool vec) {
        if (vec) r = *(const float4 *) (p + c);
        else r = make_float4(p[c], c + 1 < n ? p[c + 1] : 0.f, c + 2 < n ? p[c + 2] : 0.f, c + 3 < n ? p[c + 3] : 0.f);
    }
    __device__ __forceinline__ float4 get() const { return r; }
};
template <> struct Quad<bf16> {
    uint2 r;
    __device__ __forceinline__ void zero() { r = make_uint2(0, 0); }
    __device__ __forceinline__ void load(const bf16 * p, int c, int n, bool vec) {
        if (vec) {
            r = *(const uint2 *) (p + c);
        } else {
            const unsigned short * q = (const unsigned short *) p;
            r.x = q[c] | (c + 1 < n ? (unsigned) q[c + 1] << 16 : 0u);
            r.y = (c + 2 < n ? q[c + 2] : 0u) | (c + 3 < n ? (unsigned) q[c + 3] << 16 : 0u);
        }
    }
    __device__ __forceinline__ float4 get() const {
        const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *) &r.x), y = __bfloat1622float2(*(const __nv_bfloat162 *) &r.y);
        return make_float4(x.x, x.y, y.x, y.y);
    }
};

// What a CTA works on: rows (token i0 + r / nh of sequence b, head h0 + r % nh), r < rows, against the tiles k_lo .. k_hi of its keys: first pt
// tiles of pooled blocks (nb blocks), then the tiles of positions lo .. end, tile kt at positions (kt + t0) * KT.
struct Work {
    int b, q0, i0, g, h0, nh, rows, p0, lo, end, k_lo, k_hi, nb, pt, t0;
};
// false: no work for this CTA nor for the others of its cluster
__device__ __forceinline__ bool find_work(const jib_gqa & a, int run, int heads, int KT, Work & w) {
    // which (sequence, run of tokens)?  Sequence b's runs start at index q_start[b] / run + b; indices in the gaps have no tokens.
    // (run 0: one token per sequence)
    int b = run == 0 ? (int) blockIdx.x : 0, hi = run == 0 ? 0 : a.n_seqs;
    while (hi - b > 1) {
        const int mid = (b + hi) >> 1;
        if (a.q_start[mid] / run + mid <= (int) blockIdx.x) b = mid; else hi = mid;
    }
    w.b = b;
    w.q0 = a.q_start[b];
    const int n = a.q_start[b + 1] - w.q0;
    w.i0 = run == 0 ? 0 : ((int) blockIdx.x - (w.q0 / run + b)) * run;
    if (run == 0) run = 1;
    if (w.i0 < 0 || w.i0 >= n) return false;
    const int rep = a.H / a.G, groups = (rep + heads - 1) / heads;
    w.g = blockIdx.y / groups;
    w.h0 = w.g * rep + (blockIdx.y % groups) * heads;
    w.nh = min(heads, (w.g + 1) * rep - w.h0);
    const int nt = min(run, n - w.i0);
    w.rows = nt * w.nh;
    const int S = a.seq_lens[b];
    w.p0 = S - n + w.i0;                                     // position of the first token
    w.lo = max(0, gqa_first_key(w.p0, a.window, a.chunk));
    w.end = S > 0 ? w.p0 + nt : 0;
    w.nb = gqa_blocks_seen(w.p0 + nt - 1, a.window, a.pool_size);
    w.pt = (w.nb + KT - 1) / KT;
    const int t_lo = w.lo / KT, tiles = w.pt + (w.end > w.lo ? (w.end - 1) / KT + 1 - t_lo : 0);
    w.t0 = t_lo - w.pt;
    const int per = (tiles + (int) gridDim.z - 1) / (int) gridDim.z;
    w.k_lo = (int) blockIdx.z * per;
    w.k_hi = min(tiles, w.k_lo + per);
    return true;
}

// part [ROWS][V], m_s and l_s [ROWS] of this CTA, complete behind a barrier -> this CTA's share of the results
template <typename T>
__device__ __forceinline__ void finish_rows(const jib_gqa & a, const Work & w, const float * part, const float * m_s, const float * l_s,
                                            const T * gate, long long ld_gate, T * out, long long ldo) {
    const int n_splits = gridDim.z, V = a.V;
    if (n_splits > 1) cluster_sync(); else __syncthreads();
    for (int i = threadIdx.x + (int) blockIdx.z * NT; i < w.rows * V; i += NT * n_splits) {
        const int r = i / V, col = i % V;
        const int t = w.q0 + w.i0 + r / w.nh, h = w.h0 + r % w.nh;
        const float sink = !a.sink ? -INFINITY : a.sink_w != nullptr ? a.sink_w[h] : 0.f;
        const float gt = gate != nullptr ? to_f(gate[(size_t) t * ld_gate + (a.gate_each ? h * V + col : h)]) : 0.f;
        if (n_splits == 1) {
            const float m1 = m_s[r], m = fmaxf(sink, m1), e = m1 == -INFINITY ? 0.f : exp_t<T>(m1 - m);
            const float l = e * l_s[r] + (a.sink ? exp_t<T>(sink - m) : 0.f);
            float y = l > 0.f ? e * part[r * V + col] / l * a.out_scale : 0.f;
            if (gate != nullptr) y /= 1.f + exp_t<T>(-gt);
            put(out + (size_t) t * ldo + h * V + col, y);
            continue;
        }
        float ms[8], ls[8], os[8], m = sink;
#pragma unroll
        for (int s = 0; s < 8; ++s) {                        // every peer's value requested before any is used
            ms[s] = -INFINITY;
            ls[s] = os[s] = 0.f;
            if (s >= n_splits) continue;
            ms[s] = n_splits > 1 ? ld_peer(m_s + r, s) : m_s[r];
            ls[s] = n_splits > 1 ? ld_peer(l_s + r, s) : l_s[r];
            os[s] = n_splits > 1 ? ld_peer(part + r * V + col, s) : part[r * V + col];
        }
#pragma unroll
        for (int s = 0; s < 8; ++s) m = fmaxf(m, ms[s]);
        float l = a.sink ? exp_t<T>(sink - m) : 0.f, o = 0.f;
#pragma unroll
        for (int s = 0; s < 8; ++s) {
            const float e = ms[s] == -INFINITY ? 0.f : exp_t<T>(ms[s] - m);
            l += e * ls[s];
            o += e * os[s];
        }
        float y = l > 0.f ? o / l * a.out_scale : 0.f;
        if (gate != nullptr) y /= 1.f + exp_t<T>(-gt);
        put(out + (size_t) t * ldo + h * V + col, y);
    }
    if (n_splits > 1) cluster_sync();                        // a CTA that leaves takes its shared memory with it
}

template <typename T, int NVC>
__global__ void __launch_bounds__(NT) gqa_attention_kernel(const __grid_constant__ jib_gqa a, const T * __restrict__ q, const T * __restrict__ gate,
                                                           long long ld_gate, T * __restrict__ out, long long ldo, int run, int heads, int KT) {
    extern __shared__ float smem[];
    __shared__ int rows_s[64];
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int tid = threadIdx.x, D = a.D, V = a.V;
    const int DP = (D + 3) / 4 * 4 + 4, VP = (V + 3) / 4 * 4;
    float * qs = smem, * m_s = qs + ROWS * DP, * l_s = m_s + ROWS, * c_s = l_s + ROWS;
    float * ks = c_s + ROWS, * vs = ks + KT * DP, * ps = vs + KT * VP;                           // ps [KT][ROWS]
    Work w;
    if (!find_work(a, run, heads, KT, w)) return;
    const int q0 = w.q0, i0 = w.i0, g = w.g, h0 = w.h0, nh = w.nh, rows = w.rows, p0 = w.p0, lo = w.lo, end = w.end;
    const bool vec = ((D | V | a.row) & 3) == 0;
    for (int i = tid; i < ROWS * (DP / 4); i += NT) {
        const int r = i / (DP / 4), c = i % (DP / 4) * 4;
        float4 x = make_float4(0.f, 0.f, 0.f, 0.f);
        if (r < rows && c < D) {
            Quad<T> k;
            k.load(q + ((size_t) (q0 + i0 + r / nh) * a.H + h0 + r % nh) * D, c, D, vec);
            x = k.get();
        }
        x.x *= a.scale; x.y *= a.scale; x.z *= a.scale; x.w *= a.scale;
        *(float4 *) (qs + r * DP + c) = x;
    }
    if (tid < ROWS) { m_s[tid] = -INFINITY; l_s[tid] = 0.f; }
    float acc[NVC][ROWS];
#pragma unroll
    for (int c = 0; c < NVC; ++c)
#pragma unroll
        for (int r = 0; r < ROWS; ++r) acc[c][r] = 0.f;
    const int * bt = a.block_tables + (size_t) w.b * a.max_blocks;
    const int key = tid % KT, rg = tid / KT, rpt = ROWS * KT / NT;       // scores: this thread's key and its rpt rows
    for (int kt = w.k_lo; kt < w.k_hi; ++kt) {
        __syncthreads();
        const bool pooled = kt < w.pt;
        const int base = (pooled ? kt : kt + w.t0) * KT, first = pooled ? 0 : lo, last = pooled ? w.nb : end;      // keys first .. last - 1 exist
        const T * src = pooled ? (const T *) a.pool : (const T *) a.cache;
        if (tid < KT) {                                      // where this tile's rows are
            const int p = base + tid;
            rows_s[tid] = p >= last || p < first ? -1
                                                 : pooled ? (int) gqa_pool_row(bt, p, a.pool_size, a.pool_rows, a.block_size)
                                                          : bt[p / a.block_size] * a.block_size + p % a.block_size;
        }
        __syncthreads();
        const int k4 = DP / 4 - 1, w4 = k4 + VP / 4;
        constexpr int FLY = 8;
        for (int i = tid; i < KT * w4; i += NT * FLY) {
            Quad<T> x[FLY];
#pragma unroll
            for (int u = 0; u < FLY; ++u) {
                const int e = i + u * NT, j = e / w4, c = e - j * w4;
                x[u].zero();
                const int slot = e < KT * w4 ? rows_s[j] : -1;
                if (slot < 0) continue;
                const T * row = src + (size_t) slot * a.row;
                if (c < k4) x[u].load(row + g * D, 4 * c, D, vec);
                else x[u].load(row + a.G * D + g * V, 4 * (c - k4), V, vec);
            }
#pragma unroll
            for (int u = 0; u < FLY; ++u) {
                const int e = i + u * NT, j = e / w4, c = e - j * w4;
                if (e < KT * w4) *(float4 *) (c < k4 ? ks + j * DP + 4 * c : vs + j * VP + 4 * (c - k4)) = x[u].get();
            }
        }
        __syncthreads();
        float s[8];
#pragma unroll
        for (int r = 0; r < 8; ++r) s[r] = 0.f;
        const float * kr = ks + key * DP, * qr = qs + rg * rpt * DP;
        for (int c = 0; c < D; c += 4) {
            const float4 x = *(const float4 *) (kr + c);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                if (r >= rpt || rg * rpt + r >= rows) break;
                const float4 y = *(const float4 *) (qr + r * DP + c);
                s[r] += x.x * y.x + x.y * y.y + x.z * y.z + x.w * y.w;
            }
        }
        const int p = base + key;
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            if (r >= rpt) break;
            const int row = rg * rpt + r;
            const int pos = p0 + (row < rows ? row / nh : 0);
            const bool see = row < rows && (pooled ? p < gqa_blocks_seen(pos, a.window, a.pool_size) : p <= pos && p >= gqa_first_key(pos, a.window, a.chunk));
            const float v = a.softcap > 0.f ? capped<T>(s[r], a.softcap) : s[r];
            ps[key * ROWS + row] = see ? v : -INFINITY;
        }
        __syncthreads();
        {   // running maximum and sum: 8 lanes per row
            const int row = tid >> 3, sub = tid & 7;
            float mx = -INFINITY;
            for (int j = sub; j < KT; j += 8) mx = fmaxf(mx, ps[j * ROWS + row]);
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
            const float m_old = m_s[row], m_new = fmaxf(m_old, mx);
            float ls = 0.f;
            for (int j = sub; j < KT; j += 8) {
                const float x = ps[j * ROWS + row];
                const float e = x == -INFINITY ? 0.f : exp_t<T>(x - m_new);
                ps[j * ROWS + row] = e;
                ls += e;
            }
#pragma unroll
            for (int o = 4; o > 0; o >>= 1) ls += __shfl_xor_sync(0xffffffffu, ls, o);
            if (sub == 0) {
                const float cf = m_old == -INFINITY ? 0.f : exp_t<T>(m_old - m_new);
                c_s[row] = cf;
                m_s[row] = m_new;
                l_s[row] = l_s[row] * cf + ls;
            }
        }
        __syncthreads();
#pragma unroll
        for (int c = 0; c < NVC; ++c)
#pragma unroll
            for (int r = 0; r < ROWS; ++r) acc[c][r] *= c_s[r];
        const int jn = min(KT, last - base);
        for (int j = max(0, first - base); j < jn; ++j) {
            float pr[ROWS];
#pragma unroll
            for (int r = 0; r < ROWS; r += 4) {
                if (r >= rows) break;
                *(float4 *) (pr + r) = *(const float4 *) (ps + j * ROWS + r);
            }
#pragma unroll
            for (int c = 0; c < NVC; ++c) {
                const int col = tid + c * NT;
                const float x = col < V ? vs[j * VP + col] : 0.f;
#pragma unroll
                for (int r = 0; r < ROWS; ++r) {
                    if ((r & ~3) >= rows) break;
                    acc[c][r] += pr[r] * x;
                }
            }
        }
    }
    // partial sums [ROWS][V] where the key and value tiles were, then every CTA finishes its share of the rows
    __syncthreads();
    float * part = ks;
#pragma unroll
    for (int c = 0; c < NVC; ++c) {
        const int col = tid + c * NT;
        if (col < V)
            for (int r = 0; r < ROWS; ++r) part[r * V + col] = acc[c][r];
    }
    finish_rows<T>(a, w, part, m_s, l_s, gate, ld_gate, out, ldo);
}

// ---- attention on tensor cores: bf16, D and V multiples of 16 ---------------------------------------------------------------------
// The same decomposition; the 16 rows are the M of m16n8k16 products.  Tiles of 64 keys arrive by asynchronous copies, ST - 1 ahead; each
// of the 4 warps takes 16 keys of a tile, copies them itself (no barrier in the loop) and keeps its own running maximum, sum and output
// (NV x 8 columns), which meet at the end.
constexpr int MK = 64, PADC = 8;                             // keys per tile; padding of the shared rows (16 bytes: rows hit different banks)

__device__ __forceinline__ void mma(float (&d)[4], const uint32_t (&x)[4], uint32_t y0, uint32_t y1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(x[0]), "r"(x[1]), "r"(x[2]), "r"(x[3]), "r"(y0), "r"(y1));
}
__device__ __forceinline__ void ldm4(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ void ldm4t(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0, %1, %2, %3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr) : "memory");
}
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void cp16(uint32_t dst, const void * src, bool valid) {       // zeros if not valid (src is not read)
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(src), "r"(valid ? 16 : 0) : "memory");
}

template <int NV, int ST>                                    // columns of V per 16: V <= 16 NV; tiles in shared memory
__global__ void __launch_bounds__(NT) gqa_mma_kernel(const __grid_constant__ jib_gqa a, const bf16 * __restrict__ q, const bf16 * __restrict__ gate,
                                                     long long ld_gate, bf16 * __restrict__ out, long long ldo, int run, int heads) {
    extern __shared__ __align__(16) uint8_t smem_mma[];
    __shared__ float m_s[ROWS], l_s[ROWS], wm[4][ROWS], wl[4][ROWS];
    PDL_TRIGGER_TOP();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, D = a.D, V = a.V;
    const int LD = D + PADC, LV = V + PADC;                  // row strides (elements)
    const uint32_t q_addr = (uint32_t) __cvta_generic_to_shared(smem_mma), kv_addr = q_addr + ROWS * LD * 2;
    const uint32_t tile_bytes = MK * (LD + LV) * 2;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    Work w;
    if (!find_work(a, run, heads, MK, w)) return;
    const int * bt = a.block_tables + (size_t) w.b * a.max_blocks;
    const bf16 * cache = (const bf16 *) a.cache;
    const int d8 = D / 8, v8 = V / 8;
    // the warp's 16 keys, as 16-byte units that go round the lanes, row after row (several at a time if they are short).  16 adjacent positions
    // of a cache block follow one another; else lane l knows where key l & 15 is
    const int units = d8 + v8, at_once = units <= 32 ? 32 / units : 1, sub = units <= 32 ? lane / units : 0, unit = units <= 32 ? lane % units : lane;
    const bool whole = a.block_size % 16 == 0 && units == 32;
    auto stage = [&](int kt, int buf) {
        if (kt < w.k_hi && kt >= w.pt && whole) {
            const int p = (kt + w.t0) * MK + warp * 16;
            const bool any = p + 15 >= w.lo && p < w.end;    // else there may be no block
            const bool is_k = lane < d8;
            const int col = is_k ? w.g * D + lane * 8 : a.G * D + w.g * V + (lane - d8) * 8;
            const bf16 * src = any ? cache + ((size_t) bt[p / a.block_size] * a.block_size + p % a.block_size) * a.row + col : cache;
            uint32_t dst = kv_addr + buf * tile_bytes + (is_k ? warp * 16 * LD + lane * 8 : MK * LD + warp * 16 * LV + (lane - d8) * 8) * 2;
            const uint32_t step = (is_k ? LD : LV) * 2;
            const size_t row = any ? (size_t) a.row : 0;
#pragma unroll
            for (int r = 0; r < 16; ++r) {
                cp16(dst, src, p + r >= w.lo && p + r < w.end);
                dst += step;
                src += row;
            }
        } else if (kt < w.k_hi) {
            const bool pooled = kt < w.pt;
            const int p = (pooled ? kt : kt + w.t0) * MK + warp * 16 + (lane & 15);
            const bool in = pooled ? p < w.nb : p >= w.lo && p < w.end;
            const bf16 * row = !in ? cache
                               : pooled ? (const bf16 *) a.pool + gqa_pool_row(bt, p, a.pool_size, a.pool_rows, a.block_size) * a.row
                                        : cache + ((size_t) bt[p / a.block_size] * a.block_size + p % a.block_size) * a.row;
            const uint32_t kd = kv_addr + buf * tile_bytes + warp * 16 * LD * 2, vd = kv_addr + buf * tile_bytes + (MK * LD + warp * 16 * LV) * 2;
#pragma unroll 4
            for (int r0 = 0; r0 < 16; r0 += at_once) {
                const int r = r0 + sub;
                const bf16 * src = (const bf16 *) __shfl_sync(0xffffffffu, (unsigned long long) row, r & 15);
                const bool ok = __shfl_sync(0xffffffffu, in, r & 15);
                if (sub >= at_once || r >= 16) continue;
                for (int c = unit; c < units; c += 32) {
                    if (c < d8) cp16(kd + (r * LD + c * 8) * 2, src + w.g * D + c * 8, ok);
                    else cp16(vd + (r * LV + (c - d8) * 8) * 2, src + a.G * D + w.g * V + (c - d8) * 8, ok);
                    if (units <= 32) break;
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    for (int i = tid; i < ROWS * d8; i += NT) {
        const int r = i / d8, c = i % d8;
        cp16(q_addr + (r * LD + c * 8) * 2, q + (r < w.rows ? ((size_t) (w.q0 + w.i0 + r / w.nh) * a.H + w.h0 + r % w.nh) * D + c * 8 : 0), r < w.rows);
    }
    asm volatile("cp.async.commit_group;" ::: "memory");
#pragma unroll
    for (int i = 0; i < ST - 1; ++i) stage(w.k_lo + i, i);
    const int fr = lane >> 2, fc = (lane & 3) * 2;
    // positions, first keys and pooled blocks of this thread's two rows
    int pos[2], first[2], blocks[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int r = fr + 8 * e;
        pos[e] = r < w.rows ? w.p0 + r / w.nh : -1;
        first[e] = r < w.rows ? gqa_first_key(pos[e], a.window, a.chunk) : 0;
        blocks[e] = gqa_blocks_seen(pos[e], a.window, a.pool_size);
    }
    float o[2 * NV][4], m[2] = {-INFINITY, -INFINITY}, l[2] = {0.f, 0.f};
#pragma unroll
    for (int n = 0; n < 2 * NV; ++n)
#pragma unroll
        for (int e = 0; e < 4; ++e) o[n][e] = 0.f;
    constexpr float LOG2E = 1.4426950408889634f;
    const float sc = a.softcap > 0.f ? 2.f * LOG2E * a.scale / a.softcap : a.scale * LOG2E, cap = a.softcap * LOG2E;
    asm volatile("cp.async.wait_group %0;" ::"n"(ST - 1) : "memory");
    __syncthreads();                                         // the queries are there
    for (int kt = w.k_lo; kt < w.k_hi; ++kt) {
        const int buf = (kt - w.k_lo) % ST;
        stage(kt + ST - 1, (buf + ST - 1) % ST);
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 1) : "memory");
        __syncwarp();
        const uint32_t k_addr = kv_addr + buf * tile_bytes + warp * 16 * LD * 2, v_addr = kv_addr + buf * tile_bytes + (MK * LD + warp * 16 * LV) * 2;
        float s[2][4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) s[n][e] = 0.f;
#pragma unroll 4
        for (int kk = 0; kk < D; kk += 16) {
            uint32_t x[4], y[4];
            ldm4(x, q_addr + ((lane & 15) * LD + kk + (lane >> 4) * 8) * 2);
            ldm4(y, k_addr + (((lane & 7) + ((lane >> 4) << 3)) * LD + kk + ((lane >> 3) & 1) * 8) * 2);      // keys 0-7 | 8-15
            mma(s[0], x, y[0], y[1]);
            mma(s[1], x, y[2], y[3]);
        }
        const bool pooled = kt < w.pt;
        const int key = (pooled ? kt : kt + w.t0) * MK + warp * 16 + fc;            // this thread's keys: key, key + 1, key + 8, key + 9
        const int end[2] = {pooled ? blocks[0] : pos[0] + 1, pooled ? blocks[1] : pos[1] + 1}, from[2] = {pooled ? 0 : first[0], pooled ? 0 : first[1]};
        float mt[2] = {-INFINITY, -INFINITY};
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                float y = s[n][e] * sc;
                if (a.softcap > 0.f) {
                    float x, r;
                    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(x) : "f"(fminf(y, 120.f)));
                    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(1.f + x));
                    y = cap - 2.f * cap * r;                 // 1 - 2 / (1 + e^{2 y}) = tanh(y)
                }
                const int p = key + n * 8 + (e & 1);
                s[n][e] = p < end[e >> 1] && p >= from[e >> 1] ? y : -INFINITY;
                mt[e >> 1] = fmaxf(mt[e >> 1], s[n][e]);
            }
        float cf[2], base[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            mt[e] = fmaxf(mt[e], __shfl_xor_sync(0xffffffffu, mt[e], 1));
            mt[e] = fmaxf(mt[e], __shfl_xor_sync(0xffffffffu, mt[e], 2));
            const float mn = fmaxf(m[e], mt[e]);
            base[e] = mn == -INFINITY ? 0.f : mn;            // every score is -inf then
            cf[e] = ex2(m[e] - base[e]);
            m[e] = mn;
            l[e] *= cf[e];
        }
        uint32_t x[4];
#pragma unroll
        for (int n = 0; n < 2; ++n)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const float p0 = ex2(s[n][2 * e] - base[e]), p1 = ex2(s[n][2 * e + 1] - base[e]);
                l[e] += p0 + p1;
                const __nv_bfloat162 pk = __floats2bfloat162_rn(p0, p1);
                x[n * 2 + e] = *(const uint32_t *) &pk;
            }
#pragma unroll
        for (int n = 0; n < 2 * NV; n += 2) {
            if (n * 8 >= V) break;
            uint32_t y[4];
            ldm4t(y, v_addr + ((lane & 15) * LV + n * 8 + (lane >> 4) * 8) * 2);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                o[n][e] *= cf[e >> 1];
                o[n + 1][e] *= cf[e >> 1];
            }
            mma(o[n], x, y[0], y[1]);
            mma(o[n + 1], x, y[2], y[3]);
        }
        __syncwarp();                                        // the buffer is free
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 1);
        l[e] += __shfl_xor_sync(0xffffffffu, l[e], 2);
        if ((lane & 3) == 0) {
            wm[warp][fr + 8 * e] = m[e];
            wl[warp][fr + 8 * e] = l[e];
        }
    }
    __syncthreads();
    // the four warps' outputs, brought to a common maximum, summed in shared memory one warp after the other
    float * part = (float *) (smem_mma + ROWS * LD * 2);
    float f[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int r = fr + 8 * e;
        const float mx = fmaxf(fmaxf(wm[0][r], wm[1][r]), fmaxf(wm[2][r], wm[3][r]));
        f[e] = m[e] == -INFINITY ? 0.f : exp2f(m[e] - mx);
    }
    for (int k = 0; k < 4; ++k) {
        if (warp == k) {
#pragma unroll
            for (int n = 0; n < 2 * NV; ++n) {
                if (n * 8 >= V) break;
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float2 * p = (float2 *) (part + (fr + 8 * e) * V + n * 8 + fc);
                    float2 y = k == 0 ? make_float2(0.f, 0.f) : *p;
                    y.x += o[n][2 * e] * f[e];
                    y.y += o[n][2 * e + 1] * f[e];
                    *p = y;
                }
            }
        }
        __syncthreads();
    }
    if (tid < ROWS) {
        const float mx = fmaxf(fmaxf(wm[0][tid], wm[1][tid]), fmaxf(wm[2][tid], wm[3][tid]));
        float s = 0.f;
#pragma unroll
        for (int k = 0; k < 4; ++k) s += wm[k][tid] == -INFINITY ? 0.f : wl[k][tid] * exp2f(wm[k][tid] - mx);
        m_s[tid] = mx == -INFINITY ? mx : mx / LOG2E;        // natural units
        l_s[tid] = s;
    }
    finish_rows<bf16>(a, w, part, m_s, l_s, gate, ld_gate, out, ldo);
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

int smem_bytes(const jib_gqa & a, int KT) {
    const int DP = (a.D + 3) / 4 * 4 + 4, VP = (a.V + 3) / 4 * 4;
    int tiles = KT * (DP + VP + ROWS);
    if (tiles < ROWS * a.V) tiles = ROWS * a.V;
    return 4 * (ROWS * DP + tiles + 3 * ROWS);
}

template <typename T, int NVC>
int launch_attention(const jib_gqa & a, const void * q, const void * gate, long long ld_gate, void * out, long long ldo, int single, int splits,
                     cudaStream_t s) {
    constexpr int CAP = 200 * 1024;
    int KT = 64;
    while (KT > 8 && smem_bytes(a, KT) > CAP) KT /= 2;
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    if (smem_bytes(a, KT) > CAP || !jib::ensure_dyn_smem(gqa_attention_kernel<T, NVC>, CAP, done)) return JIB_E_ARG;
    const int rep = a.H / a.G, heads = rep < ROWS ? rep : ROWS, run = single ? 0 : ROWS / heads;
    const dim3 grid(single ? a.T : a.T / run + a.n_seqs, a.G * ((rep + heads - 1) / heads), splits);
    const cudaError_t e = jib::launch_pdl_cluster(gqa_attention_kernel<T, NVC>, grid, dim3(NT), (size_t) smem_bytes(a, KT), s, splits, a, (const T *) q,
                                                  (const T *) gate, ld_gate, (T *) out, ldo, run, heads, KT);
    if (e != cudaSuccess) { (void) cudaGetLastError(); return JIB_E_LAUNCH; }
    return launched();
}

// bf16 rows that 16-byte copies can address
bool mma_ok(const jib_gqa & a, const void * q) {
    return a.D % 16 == 0 && a.V % 16 == 0 && a.V <= 256 && a.row % 8 == 0 && (((uintptr_t) a.cache | (uintptr_t) a.pool | (uintptr_t) q) & 15) == 0;
}

template <int NV, int ST>
int launch_mma_as(const jib_gqa & a, const void * q, const void * gate, long long ld_gate, void * out, long long ldo, int single, int splits,
                  cudaStream_t s) {
    const int tile = MK * (a.D + a.V + 2 * PADC) * 2, smem = ROWS * (a.D + PADC) * 2 + ST * tile;       // >= the [ROWS][V] partial results
    constexpr int CAP = 220 * 1024;
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    if (smem > CAP || !jib::ensure_dyn_smem(gqa_mma_kernel<NV, ST>, CAP, done)) return JIB_E_ARG;
    const int rep = a.H / a.G, heads = rep < ROWS ? rep : ROWS, run = single ? 0 : ROWS / heads;
    const dim3 grid(single ? a.T : a.T / run + a.n_seqs, a.G * ((rep + heads - 1) / heads), splits);
    const cudaError_t e = jib::launch_pdl_cluster(gqa_mma_kernel<NV, ST>, grid, dim3(NT), (size_t) smem, s, splits, a, (const bf16 *) q, (const bf16 *) gate,
                                                  ld_gate, (bf16 *) out, ldo, run, heads);
    if (e != cudaSuccess) { (void) cudaGetLastError(); return JIB_E_LAUNCH; }
    return launched();
}

// Three tiles in shared memory while two CTAs fit on an SM; two where the keys are split over CTAs that have one or two tiles each
template <int NV>
int launch_mma(const jib_gqa & a, const void * q, const void * gate, long long ld_gate, void * out, long long ldo, int single, int splits,
               cudaStream_t s) {
    const int smem = ROWS * (a.D + PADC) * 2 + 3 * MK * (a.D + a.V + 2 * PADC) * 2;
    return smem <= 112 * 1024 && splits == 1 ? launch_mma_as<NV, 3>(a, q, gate, ld_gate, out, ldo, single, splits, s)
                              : launch_mma_as<NV, 2>(a, q, gate, ld_gate, out, ldo, single, splits, s);
}

// Whole vectors of 4 in every row that gqa_pairs_post reads and writes
bool pairs_ok(const jib_gqa & a, const void * q, const void * k, const void * v, long long ld, const void * q_out, int el) {
    const uintptr_t at = (uintptr_t) q | (uintptr_t) k | (uintptr_t) v | (uintptr_t) q_out | (uintptr_t) a.cache | (uintptr_t) a.v_first;
    const long long n = a.D | a.V | ld | a.row | (a.mix_v ? a.ld_first : 0);
    return at % (4 * el) == 0 && n % 4 == 0 && a.D <= 512 && a.V <= 512;
}

int launch_pool(const jib_gqa & a, int f32, cudaStream_t s) {
    if (a.q_start == nullptr || a.seq_lens == nullptr || a.n_seqs <= 0) return JIB_E_ARG;
    const int e = f32 ? 4 : 8, cols = a.G * (a.D + a.V), n = a.T / a.pool_size + a.n_seqs;
    if (cols % e == 0 && a.row % e == 0 && (((uintptr_t) a.cache | (uintptr_t) a.pool) & 15) == 0) {
        const dim3 grid(n, (cols / e + 31) / 32);
        if (f32) JIB_LAUNCH((gqa_pool_vec_kernel<float>), grid, 256, 0, s, a);
        else JIB_LAUNCH((gqa_pool_vec_kernel<bf16>), grid, 256, 0, s, a);
        return launched();
    }
    if (f32) JIB_LAUNCH((gqa_pool_kernel<float>), n, 256, 0, s, a);
    else JIB_LAUNCH((gqa_pool_kernel<bf16>), n, 256, 0, s, a);
    return launched();
}

bool ok(const jib_gqa & a) {
    return a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.D >= 1 && a.D <= 32 * POST_D && a.V >= 1 && a.V <= 4 * NT && a.rot >= 0 && a.rot % 2 == 0 && a.rot <= a.D &&
           a.row >= (long long) a.G * (a.D + a.V) && a.T <= 65535 && a.block_size > 0 &&
           (a.pool_size == 0 || (a.pool_size > 0 && a.window > 0 && a.pool != nullptr && a.block_tables != nullptr &&
                                 a.pool_rows >= (a.block_size + a.pool_size - 1) / a.pool_size));
}

}  // namespace

extern "C" {

JIB_EXPORT int jib_gqa_qkv_post(const jib_gqa * m, const void * q, const void * k, const void * v, long long ld, const float * q_norm,
                                const float * k_norm, const float * rope, const int * slot_mapping, void * q_out, int single, int f32, void * stream) {
    const jib_gqa & a = *m;
    if (a.T <= 0) return 0;
    if (!ok(a) || (a.mix_v && a.v_first == nullptr) || (single && a.pool_size > 0 && a.n_seqs != a.T)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    const int el = f32 ? 4 : 2;
    const bool pool = a.pool_size > 0;
    if (a.neighbours && q_norm == nullptr && k_norm == nullptr && !(single && pool) && pairs_ok(a, q, k, v, ld, q_out, el)) {
        const int n = a.D > a.V ? a.D : a.V, tok = a.T >= 256 && n <= 256 ? 2 : 1;
        const dim3 grid((a.H + 2 * a.G + 7) / 8, (a.T + tok - 1) / tok);
#define PAIRS(TT, N, TOK) \
    JIB_LAUNCH((gqa_pairs_post_kernel<TT, N, TOK>), grid, 256, 0, s, a, (const TT *) q, (const TT *) k, (const TT *) v, ld, rope, slot_mapping, (TT *) q_out)
#define CALL(N, TOK)                    \
    do {                                \
        if (f32) PAIRS(float, N, TOK);  \
        else PAIRS(bf16, N, TOK);       \
    } while (0)
        if (n <= 128 && tok == 2) CALL(1, 2);
        else if (n <= 128) CALL(1, 1);
        else if (n <= 256 && tok == 2) CALL(2, 2);
        else if (n <= 256) CALL(2, 1);
        else CALL(4, 1);
#undef CALL
#undef PAIRS
        const int rc = launched();
        return rc || !pool ? rc : launch_pool(a, f32, s);
    }
    const dim3 grid((a.H + 2 * a.G + 7) / 8, a.T);
    const int smem = 8 * a.D * 4;
#define POST(TT, N)                                                                                                                        \
    JIB_LAUNCH((gqa_qkv_post_kernel<TT, N>), grid, 256, smem, s, a, (const TT *) q, (const TT *) k, (const TT *) v, ld, q_norm, k_norm, rope, \
               slot_mapping, (TT *) q_out, single)
#define CALL(N)                     \
    do {                            \
        if (f32) POST(float, N);    \
        else POST(bf16, N);         \
    } while (0)
    if (a.D <= 64) CALL(2);
    else if (a.D <= 128) CALL(4);
    else CALL(POST_D);
#undef CALL
#undef POST
    const int rc = launched();
    return rc || single || !pool ? rc : launch_pool(a, f32, s);
}

JIB_EXPORT int jib_gqa_attention(const jib_gqa * m, const void * q, const void * gate, long long ld_gate, void * out, long long ldo, int single,
                                 int splits, int f32, void * stream) {
    const jib_gqa & a = *m;
    if (a.T <= 0 || a.n_seqs <= 0) return 0;
    if (!ok(a) || splits < 1 || splits > 8 || (single && a.T != a.n_seqs)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    if (!f32 && mma_ok(a, q)) {
        if (a.V <= 64) return launch_mma<4>(a, q, gate, ld_gate, out, ldo, single, splits, s);
        if (a.V <= 128) return launch_mma<8>(a, q, gate, ld_gate, out, ldo, single, splits, s);
        return launch_mma<16>(a, q, gate, ld_gate, out, ldo, single, splits, s);
    }
#define CALL(NVC) (f32 ? launch_attention<float, NVC>(a, q, gate, ld_gate, out, ldo, single, splits, s)     \
                       : launch_attention<bf16, NVC>(a, q, gate, ld_gate, out, ldo, single, splits, s))
    if (a.V <= NT) return CALL(1);
    if (a.V <= 2 * NT) return CALL(2);
    return CALL(4);
#undef CALL
}

}  // extern "C"
