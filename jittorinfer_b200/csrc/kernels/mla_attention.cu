// Weight-absorbed MLA attention over the paged latent cache, split-KV ("flash-decoding") form.
//
// The reference composes this from four matmuls and a softmax that materialise [S, T*H] scores in HBM and
// keeps a second, transposed copy of the latent (src/llama-graph-attn.cpp:219-342); its mask is a dense
// host-built [n_kv x T] matrix (src/llama-context.cpp:326-423).  Here one kernel streams each latent row
// once per (token, head-group, kv-split), keeps scores on chip, derives causality from sequence lengths,
// and a small second kernel merges the split partials (m, l, o).
//
// This file is the CUDA-core (SIMT) implementation: any latent / RoPE width and head count, any q_len, bf16 or fp32 rows,
// optionally a sliding window (position i sees j with 0 <= i - j < window).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <float.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "pdl.cuh"
#include "timeline.cuh"

namespace {

typedef __nv_bfloat16 bf16;

constexpr int HG = 16;        // heads per block
constexpr int PC = 32;        // kv positions per chunk
constexpr int NT = 256;

__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ void put(bf16 * p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void put(float * p, float v) { *p = v; }
template <typename T> __device__ __forceinline__ float exp_t(float x);      // fp32 rows: the accurate function
template <> __device__ __forceinline__ float exp_t<bf16>(float x) { return __expf(x); }
template <> __device__ __forceinline__ float exp_t<float>(float x) { return expf(x); }

// Floats per staged row: a multiple of 4 whose quarter is odd, so that 16-byte reads of different rows hit different banks.
__host__ __device__ inline int row_floats(int D) {
    const int q = (D + 3) / 4;
    return 4 * (q | 1);
}
__host__ __device__ inline size_t attn_smem(int D) { return ((size_t) (HG + PC) * row_floats(D) + HG * PC) * sizeof(float); }

// One 16-byte vector of a row (8 bf16 or 4 fp32), or element by element where rows are not 16-byte multiples.
__device__ __forceinline__ void stage_row(const bf16 * src, float * dst, int D, int lane, int n_lanes, float mul) {
    if ((D & 7) == 0) {
        for (int v = lane; v < D / 8; v += n_lanes) {
            const uint4 raw = ((const uint4 *) src)[v];
            const __nv_bfloat162 * p = (const __nv_bfloat162 *) &raw;
            const float2 a = __bfloat1622float2(p[0]), b = __bfloat1622float2(p[1]), c = __bfloat1622float2(p[2]), d = __bfloat1622float2(p[3]);
            ((float4 *) dst)[2 * v] = make_float4(a.x * mul, a.y * mul, b.x * mul, b.y * mul);
            ((float4 *) dst)[2 * v + 1] = make_float4(c.x * mul, c.y * mul, d.x * mul, d.y * mul);
        }
    } else {
        for (int i = lane; i < D; i += n_lanes) dst[i] = __bfloat162float(src[i]) * mul;
    }
}
__device__ __forceinline__ void stage_row(const float * src, float * dst, int D, int lane, int n_lanes, float mul) {
    for (int i = lane; i < D; i += n_lanes) dst[i] = src[i] * mul;
}

// grid: (T, n_splits, ceil(H/HG)).  part_o [T][n_splits][H][r] (unnormalised), part_ml [T][n_splits][H][2].
// RMAX >= r bounds the accumulator registers (RMAX / 16 per thread); r, dr are the real widths.
template <typename T, int RMAX>
__global__ void __launch_bounds__(NT) mla_attn_split_kernel(const T * __restrict__ q, const T * __restrict__ cache,
                                                            const int * __restrict__ block_tables, int max_blocks,
                                                            const int * __restrict__ seq_lens, const int * __restrict__ q_start, int n_seqs,
                                                            int H, int r, int dr, int block_size, float scale, int window, int n_splits,
                                                            float * __restrict__ part_o, float * __restrict__ part_ml,
                                                            T * __restrict__ o_lat) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int D = r + dr;
    const int RS = row_floats(D);
    extern __shared__ __align__(16) float smem_f[];
    float * qs = smem_f;                       // [HG][RS]
    float * lat = qs + HG * RS;                // [PC][RS]
    float * ps = lat + PC * RS;                // [HG][PC]
    const int t = blockIdx.x, sp = blockIdx.y, hg = blockIdx.z;
    const int tid = threadIdx.x;

    // which sequence owns token t (q_start is ascending)
    int lo = 0, hi = n_seqs;
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (q_start[mid] <= t) lo = mid; else hi = mid;
    }
    const int b = lo;
    const int q0 = q_start[b], q1 = q_start[b + 1];
    const int S = seq_lens[b];
    const int n_kv = (t < q1 && S > 0) ? S - (q1 - q0) + (t - q0) + 1 : 0;   // causal: positions [0, pos]
    const int first = window > 0 ? max(0, n_kv - window) : 0;                // sliding window: positions [first, pos]
    int chunk = (n_kv - first + n_splits - 1) / n_splits;
    chunk = (chunk + PC - 1) / PC * PC;
    if (chunk < 2 * PC) chunk = 2 * PC;
    const int k0 = first + sp * chunk;
    const int k1 = min(n_kv, k0 + chunk);

    const int h_local = tid >> 4;           // 0..15 : head inside the group
    const int sub = tid & 15;
    const int h = hg * HG + h_local;
    const size_t pidx = ((size_t) t * n_splits + sp) * H + h;

    if (k0 >= k1) {
        if (n_splits > 1) {
            if (sub == 0 && h < H) { part_ml[pidx * 2] = -INFINITY; part_ml[pidx * 2 + 1] = 0.f; }
        } else {
            for (int i = sub; i < r && h < H; i += 16) put(o_lat + ((size_t) t * H + h) * r + i, 0.f);
        }
        return;
    }

    // the padding floats behind each row are never written by the staging below: zero them once
    for (int i = tid; i < (HG + PC) * (RS - D); i += NT) qs[(i / (RS - D)) * RS + D + i % (RS - D)] = 0.f;
    if (h < H) {
        stage_row(q + ((size_t) t * H + h) * D, qs + h_local * RS, D, sub, 16, scale);
    } else {
        for (int i = sub; i < D; i += 16) qs[h_local * RS + i] = 0.f;
    }

    float4 acc[RMAX / 64];                  // dims 4 * (sub + 16 * i) .. + 3
#pragma unroll
    for (int i = 0; i < RMAX / 64; ++i) acc[i] = make_float4(0.f, 0.f, 0.f, 0.f);
    float m_run = -INFINITY, l_run = 0.f;
    const int * bt = block_tables + (size_t) b * max_blocks;
    const int nv4 = (D + 3) / 4;

    for (int c0 = k0; c0 < k1; c0 += PC) {
        __syncthreads();
        for (int j = h_local; j < PC; j += NT / 16) {        // 16 lanes per row
            const int p = c0 + j;
            if (p < k1) {
                const int blk = bt[p / block_size];
                stage_row(cache + ((size_t) blk * block_size + p % block_size) * D, lat + j * RS, D, sub, 16, 1.f);
            } else {
                for (int i = sub; i < D; i += 16) lat[j * RS + i] = 0.f;
            }
        }
        __syncthreads();
        // scores: thread (h_local, sub) -> positions sub and sub+16
        float s0 = 0.f, s1 = 0.f;
        {
            const float4 * qh = (const float4 *) (qs + h_local * RS);
            const float4 * r0 = (const float4 *) (lat + sub * RS);
            const float4 * r1 = (const float4 *) (lat + (sub + 16) * RS);
#pragma unroll 4
            for (int v = 0; v < nv4; ++v) {
                const float4 a = r0[v], c = r1[v], w = qh[v];
                s0 += a.x * w.x + a.y * w.y + a.z * w.z + a.w * w.w;
                s1 += c.x * w.x + c.y * w.y + c.z * w.z + c.w * w.w;
            }
        }
        if (c0 + sub >= k1) s0 = -INFINITY;
        if (c0 + sub + 16 >= k1) s1 = -INFINITY;
        float mx = fmaxf(s0, s1);
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, o));
        const float m_new = fmaxf(m_run, mx);
        const float p0 = exp_t<T>(s0 - m_new), p1 = exp_t<T>(s1 - m_new);
        float ls = p0 + p1;
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) ls += __shfl_xor_sync(0xffffffffu, ls, o);
        const float corr = exp_t<T>(m_run - m_new);
        l_run = l_run * corr + ls;
        m_run = m_new;
        ps[h_local * PC + sub] = p0;
        ps[h_local * PC + sub + 16] = p1;
#pragma unroll
        for (int i = 0; i < RMAX / 64; ++i) { acc[i].x *= corr; acc[i].y *= corr; acc[i].z *= corr; acc[i].w *= corr; }
        __syncwarp();
        // o += p * c
        const float * ph = ps + h_local * PC;
#pragma unroll 2
        for (int j = 0; j < PC; ++j) {
            const float pj = ph[j];
            const float4 * rowp = (const float4 *) (lat + j * RS);
#pragma unroll
            for (int i = 0; i < RMAX / 64; ++i) {
                if (4 * (sub + 16 * i) < r) {
                    const float4 f = rowp[sub + 16 * i];
                    acc[i].x += pj * f.x; acc[i].y += pj * f.y; acc[i].z += pj * f.z; acc[i].w += pj * f.w;
                }
            }
        }
    }

    if (h >= H) return;                     // padding head of a partial head group: nothing to store
    const bool split = n_splits > 1;
    const float inv = l_run > 0.f ? 1.f / l_run : 0.f;
#pragma unroll
    for (int i = 0; i < RMAX / 64; ++i) {
        const float v[4] = {acc[i].x, acc[i].y, acc[i].z, acc[i].w};
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int dim = 4 * (sub + 16 * i) + e;
            if (dim >= r) continue;
            if (split) part_o[pidx * r + dim] = v[e];
            else put(o_lat + ((size_t) t * H + h) * r + dim, v[e] * inv);
        }
    }
    if (split && sub == 0) { part_ml[pidx * 2] = m_run; part_ml[pidx * 2 + 1] = l_run; }
}

// grid (T, H); 128 threads. Merges split partials.
template <typename T>
__device__ __noinline__ void mla_combine_head(const float * __restrict__ part_o, const float * __restrict__ part_ml, int n_splits, int H,
                                              int r, T * __restrict__ o_lat, float * wsm, bool dry) {
    // n_splits <= 32: warp 0 turns the (m, l) pairs into normalised weights, then every thread sums its
    // dims over the splits with independent loads.  dry: same instructions, no stores (see pdl.cuh: warm_enabled).
    const int t = blockIdx.x, h = blockIdx.y;
    if (threadIdx.x < 32) {
        const int s = threadIdx.x;
        float m = -INFINITY, l = 0.f;
        if (s < n_splits) {
            const size_t pidx = ((size_t) t * n_splits + s) * H + h;
            m = part_ml[pidx * 2];
            l = part_ml[pidx * 2 + 1];
        }
        float M = m;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
        const float w = (l > 0.f && M > -INFINITY) ? exp_t<T>(m - M) : 0.f;
        float L = l * w;
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
        wsm[s] = L > 0.f ? w / L : 0.f;
    }
    __syncthreads();
    if ((r & 3) == 0) {
        // float4 per thread, 8 splits unrolled: enough independent loads in flight to cover L2 latency
        for (int i = threadIdx.x * 4; i < r; i += blockDim.x * 4) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll 8
            for (int s = 0; s < n_splits; ++s) {
                const float w = wsm[s];
                const float4 v = *(const float4 *) (part_o + (((size_t) t * n_splits + s) * H + h) * r + i);
                if (w > 0.f) {                       // empty splits never wrote part_o
                    acc.x += w * v.x; acc.y += w * v.y; acc.z += w * v.z; acc.w += w * v.w;
                }
            }
            alignas(16) T o[4];
            put(o, acc.x); put(o + 1, acc.y); put(o + 2, acc.z); put(o + 3, acc.w);
            if (!dry) {
                T * po = o_lat + ((size_t) t * H + h) * r + i;
                if (sizeof(T) == 2) *(uint2 *) po = *(const uint2 *) o;
                else *(uint4 *) po = *(const uint4 *) o;
            }
        }
    } else {
        for (int i = threadIdx.x; i < r; i += blockDim.x) {
            float acc = 0.f;
            for (int s = 0; s < n_splits; ++s)
                if (wsm[s] > 0.f) acc += wsm[s] * part_o[(((size_t) t * n_splits + s) * H + h) * r + i];
            if (!dry) put(o_lat + ((size_t) t * H + h) * r + i, acc);
        }
    }
    __syncthreads();
}

template <typename T>
__global__ void mla_attn_combine_kernel(const float * __restrict__ part_o, const float * __restrict__ part_ml, int n_splits, int H, int r,
                                        T * __restrict__ o_lat, int warm) {
    JIB_KS(3, 0);
    PDL_TRIGGER_TOP();
    __shared__ float wsm[32];
    if (warm) mla_combine_head<T>(part_o, part_ml, n_splits, H, r, o_lat, wsm, true);
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    JIB_KS(3, 1);
    mla_combine_head<T>(part_o, part_ml, n_splits, H, r, o_lat, wsm, false);
    JIB_KS(3, 9);
}

template <typename T, int RMAX>
int launch_attn(const void * q, const void * cache, const int * block_tables, int max_blocks, const int * seq_lens, const int * q_start,
                int n_seqs, int tokens, int H, int r, int dr, int block_size, float scale, int window, int n_splits, float * part_o,
                float * part_ml, void * o_lat, cudaStream_t s) {
    const size_t smem = attn_smem(r + dr);
    if (smem > 227 * 1024) return JIB_E_ARG;
    static std::atomic<unsigned char> attr_done[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(mla_attn_split_kernel<T, RMAX>, 227 * 1024, attr_done)) return JIB_E_LAUNCH;
    JIB_LAUNCH((mla_attn_split_kernel<T, RMAX>), dim3(tokens, n_splits, (H + HG - 1) / HG), NT, smem, s, (const T *) q, (const T *) cache,
               block_tables, max_blocks, seq_lens, q_start, n_seqs, H, r, dr, block_size, scale, window, n_splits, part_o, part_ml,
               (T *) o_lat);
    if (cudaGetLastError() != cudaSuccess) return JIB_E_LAUNCH;
    if (n_splits > 1)
        JIB_LAUNCH((mla_attn_combine_kernel<T>), dim3(tokens, H), 128, 0, s, part_o, part_ml, n_splits, H, r, (T *) o_lat, jib::warm_for(tokens));
    return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH;
}

}  // namespace

JIB_TL_DEFINE_SETTER(attn)

extern "C" int jib_mla_attention(const void * q, const void * cache, const int * block_tables, int max_blocks, const int * seq_lens,
                                 const int * q_start, int n_seqs, int T, int H, int r, int dr, int block_size, float scale, int window,
                                 int n_splits, int f32, float * part_o, float * part_ml, void * o_lat, void * stream) {
    if (T <= 0) return 0;
    if (n_splits < 1 || n_splits > 32 || r < 1 || dr < 0 || block_size < 1) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
#define JIB_MLA_CASE(RMAX)                                                                                                            \
    if (r <= RMAX)                                                                                                                     \
        return f32 ? launch_attn<float, RMAX>(q, cache, block_tables, max_blocks, seq_lens, q_start, n_seqs, T, H, r, dr, block_size,  \
                                              scale, window, n_splits, part_o, part_ml, o_lat, s)                                      \
                   : launch_attn<bf16, RMAX>(q, cache, block_tables, max_blocks, seq_lens, q_start, n_seqs, T, H, r, dr, block_size,   \
                                             scale, window, n_splits, part_o, part_ml, o_lat, s);
    JIB_MLA_CASE(64)
    JIB_MLA_CASE(128)
    JIB_MLA_CASE(256)
    JIB_MLA_CASE(512)
    JIB_MLA_CASE(1024)
#undef JIB_MLA_CASE
    return JIB_E_ARG;
}

// Merge of split-KV partials (m, l, o) written by either attention kernel (bf16 result).
extern "C" int jib_mla_combine(const float * part_o, const float * part_ml, int n_splits, int T, int H, int r, void * o_lat,
                               void * stream) {
    if (T <= 0) return 0;
    if (n_splits < 1 || n_splits > 32 || r < 1) return JIB_E_ARG;
    JIB_LAUNCH((mla_attn_combine_kernel<bf16>), dim3(T, H), 128, 0, (cudaStream_t) stream, part_o, part_ml, n_splits, H, r, (bf16 *) o_lat,
               jib::warm_for(T));
    return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH;
}
