// Grouped-query attention over paged key / value rows: H query heads share G key / value heads (head h reads h / (H / G)).
// A cached row holds the normed and rotated keys of a token (G * D columns), then its values (G * V columns).
//
//   gqa_qkv_post    per-head RMS norm of q and k, rotate-half RoPE on the first rot dimensions, rows into the cache
//   gqa_attention   scores * scale, softcap, causal mask with a sliding window and / or chunks counted from position 0, softmax
//                   with or without a sink (a key of score 0 without a value), a gate per head: any sizes, any mix of portions
//                   and single tokens, keys split over a thread-block cluster
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

// ---- norm, rotation, cache rows: one warp per (token, head of q / k / v) ------------------------------------------------------
constexpr int POST_D = 16;                                   // elements of a head per lane: D <= 32 * POST_D

template <typename T>
__global__ void __launch_bounds__(256) gqa_qkv_post_kernel(const __grid_constant__ jib_gqa a, const T * __restrict__ q, const T * __restrict__ k,
                                                           const T * __restrict__ v, long long ld, const float * __restrict__ q_norm,
                                                           const float * __restrict__ k_norm, const float * __restrict__ rope,
                                                           const int * __restrict__ slot_mapping, T * __restrict__ q_out) {
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
    if (item >= H + G) {
        const int g = item - H - G;
        const T * src = v + (size_t) t * ld + g * V;
        T * dst = row + G * D + g * V;
        for (int c = lane; c < V; c += 32) dst[c] = src[c];
        return;
    }
    const bool is_q = item < H;
    const int head = is_q ? item : item - H;
    const T * src = (is_q ? q : k) + (size_t) t * ld + head * D;
    const float * w = is_q ? q_norm : k_norm;
    float * x = heads + warp * D;
    float e[POST_D], ss = 0.f;
#pragma unroll
    for (int i = 0; i < POST_D; ++i) {
        const int c = lane + 32 * i;
        e[i] = c < D ? to_f(src[c]) : 0.f;
        ss += e[i] * e[i];
    }
    const float inv = rsqrtf(warp_sum(ss) / (float) D + a.eps);
#pragma unroll
    for (int i = 0; i < POST_D; ++i) {
        const int c = lane + 32 * i;
        if (c < D) x[c] = e[i] * inv * w[c];
    }
    __syncwarp();
    int pos = a.positions[t];
    if (pos < 0 || pos >= a.max_pos) {
        if (lane == 0) jib_report(a.status, JIB_ERR_BOUNDS, 49, pos);
        pos = 0;
    }
    const float2 * cs = (const float2 *) rope + (size_t) pos * (a.rot / 2);
    T * dst = is_q ? q_out + ((size_t) t * H + head) * D : row + head * D;
    const int half = a.rot / 2;
    for (int c = lane; c < D; c += 32) {
        float y = x[c];
        if (c < half) y = y * cs[c].x - x[c + half] * cs[c].y;
        else if (c < a.rot) y = y * cs[c - half].x + x[c - half] * cs[c - half].y;
        put(dst + c, y);
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

template <typename T, int NVC>
__global__ void __launch_bounds__(NT) gqa_attention_kernel(const __grid_constant__ jib_gqa a, const T * __restrict__ q, const T * __restrict__ gate,
                                                           long long ld_gate, T * __restrict__ out, long long ldo, int run, int heads, int KT) {
    extern __shared__ float smem[];
    __shared__ int rows_s[64];
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int tid = threadIdx.x, D = a.D, V = a.V, rep = a.H / a.G;
    const int DP = (D + 3) / 4 * 4 + 4, VP = (V + 3) / 4 * 4;
    float * qs = smem, * m_s = qs + ROWS * DP, * l_s = m_s + ROWS, * c_s = l_s + ROWS;
    float * ks = c_s + ROWS, * vs = ks + KT * DP, * ps = vs + KT * VP;                           // ps [KT][ROWS]
    // which (sequence, run of tokens)?  Sequence b's runs start at index q_start[b] / run + b; indices in the gaps have no tokens.
    // (run 0: one token per sequence)
    int b = run == 0 ? (int) blockIdx.x : 0, hi = run == 0 ? 0 : a.n_seqs;
    while (hi - b > 1) {
        const int mid = (b + hi) >> 1;
        if (a.q_start[mid] / run + mid <= (int) blockIdx.x) b = mid; else hi = mid;
    }
    const int q0 = a.q_start[b], n = a.q_start[b + 1] - q0, i0 = run == 0 ? 0 : ((int) blockIdx.x - (q0 / run + b)) * run;
    if (run == 0) run = 1;
    if (i0 < 0 || i0 >= n) return;                           // the same for the whole cluster
    const int groups = (rep + heads - 1) / heads, g = blockIdx.y / groups, h0 = g * rep + (blockIdx.y % groups) * heads;
    const int nh = min(heads, (g + 1) * rep - h0), nt = min(run, n - i0), rows = nt * nh;       // row r: token i0 + r / nh, head h0 + r % nh
    const int S = a.seq_lens[b], p0 = S - n + i0;            // position of the first token
    const int lo = max(0, gqa_first_key(p0, a.window, a.chunk)), end = S > 0 ? p0 + nt : 0;
    const int t_lo = lo / KT, tiles = end > lo ? (end - 1) / KT + 1 - t_lo : 0;
    const int split = blockIdx.z, n_splits = gridDim.z, per = (tiles + n_splits - 1) / n_splits;
    const int k_lo = t_lo + split * per, k_hi = min(t_lo + tiles, k_lo + per);
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
    const int * bt = a.block_tables + (size_t) b * a.max_blocks;
    const int key = tid % KT, rg = tid / KT, rpt = ROWS * KT / NT;       // scores: this thread's key and its rpt rows
    for (int kt = k_lo; kt < k_hi; ++kt) {
        __syncthreads();
        if (tid < KT) {                                      // where this tile's rows are
            const int p = kt * KT + tid;
            rows_s[tid] = p < end && p >= lo ? bt[p / a.block_size] * a.block_size + p % a.block_size : -1;
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
                const T * row = (const T *) a.cache + (size_t) slot * a.row;
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
        const int p = kt * KT + key;
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            if (r >= rpt) break;
            const int row = rg * rpt + r;
            const int pos = p0 + (row < rows ? row / nh : 0);
            const bool see = row < rows && p <= pos && p >= gqa_first_key(pos, a.window, a.chunk);
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
        const int jn = min(KT, end - kt * KT);
        for (int j = max(0, lo - kt * KT); j < jn; ++j) {
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
    if (n_splits > 1) cluster_sync(); else __syncthreads();
    for (int i = tid + split * NT; i < rows * V; i += NT * n_splits) {
        const int r = i / V, col = i % V;
        float m = a.sink ? 0.f : -INFINITY;
        for (int s = 0; s < n_splits; ++s) m = fmaxf(m, n_splits > 1 ? ld_peer(m_s + r, s) : m_s[r]);
        float l = a.sink ? exp_t<T>(-m) : 0.f, o = 0.f;
        for (int s = 0; s < n_splits; ++s) {
            const float ms = n_splits > 1 ? ld_peer(m_s + r, s) : m_s[r];
            if (ms == -INFINITY) continue;
            const float w = exp_t<T>(ms - m);
            l += w * (n_splits > 1 ? ld_peer(l_s + r, s) : l_s[r]);
            o += w * (n_splits > 1 ? ld_peer(part + r * V + col, s) : part[r * V + col]);
        }
        const int t = q0 + i0 + r / nh, h = h0 + r % nh;
        float y = l > 0.f ? o / l * a.out_scale : 0.f;
        if (gate != nullptr) y /= 1.f + exp_t<T>(-to_f(gate[(size_t) t * ld_gate + h]));
        put(out + (size_t) t * ldo + h * V + col, y);
    }
    if (n_splits > 1) cluster_sync();                        // a CTA that leaves takes its shared memory with it
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

bool ok(const jib_gqa & a) {
    return a.H >= 1 && a.G >= 1 && a.H % a.G == 0 && a.D >= 1 && a.D <= 32 * POST_D && a.V >= 1 && a.V <= 4 * NT && a.rot >= 0 && a.rot % 2 == 0 && a.rot <= a.D &&
           a.row >= (long long) a.G * (a.D + a.V) && a.T <= 65535 && a.block_size > 0;
}

}  // namespace

extern "C" {

JIB_EXPORT int jib_gqa_qkv_post(const jib_gqa * m, const void * q, const void * k, const void * v, long long ld, const float * q_norm,
                                const float * k_norm, const float * rope, const int * slot_mapping, void * q_out, int f32, void * stream) {
    const jib_gqa & a = *m;
    if (a.T <= 0) return 0;
    if (!ok(a)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    const dim3 grid((a.H + 2 * a.G + 7) / 8, a.T);
    const int smem = 8 * a.D * 4;
    if (f32)
        JIB_LAUNCH((gqa_qkv_post_kernel<float>), grid, 256, smem, s, a, (const float *) q, (const float *) k, (const float *) v, ld, q_norm, k_norm,
                   rope, slot_mapping, (float *) q_out);
    else
        JIB_LAUNCH((gqa_qkv_post_kernel<bf16>), grid, 256, smem, s, a, (const bf16 *) q, (const bf16 *) k, (const bf16 *) v, ld, q_norm, k_norm, rope,
                   slot_mapping, (bf16 *) q_out);
    return launched();
}

JIB_EXPORT int jib_gqa_attention(const jib_gqa * m, const void * q, const void * gate, long long ld_gate, void * out, long long ldo, int single,
                                 int splits, int f32, void * stream) {
    const jib_gqa & a = *m;
    if (a.T <= 0 || a.n_seqs <= 0) return 0;
    if (!ok(a) || splits < 1 || splits > 8 || (single && a.T != a.n_seqs)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
#define CALL(NVC) (f32 ? launch_attention<float, NVC>(a, q, gate, ld_gate, out, ldo, single, splits, s)     \
                       : launch_attention<bf16, NVC>(a, q, gate, ld_gate, out, ldo, single, splits, s))
    if (a.V <= NT) return CALL(1);
    if (a.V <= 2 * NT) return CALL(2);
    return CALL(4);
#undef CALL
}

}  // extern "C"
