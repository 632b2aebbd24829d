// Mechanisms with a per-sequence state instead of a paged cache: a short causal convolution over time and a gated
// recurrence.  A sequence's state lives in row seq_slots[b] of a [n_state, ...] tensor; a batch row range that starts at
// position 0 starts from zeros whatever the row holds, so rows are handed from one sequence to the next without clearing.
// Sequence b owns token rows q_start[b] .. q_start[b + 1] of the batch (prompt portions and single tokens alike).
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "pdl.cuh"
#include "sm100.cuh"

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ void put(bf16 * p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void put(float * p, float v) { *p = v; }
__device__ __forceinline__ void load4(const float * p, float (&v)[4]) {
    const float4 a = *(const float4 *) p;
    v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w;
}
__device__ __forceinline__ void load4(const bf16 * p, float (&v)[4]) {
    const uint2 raw = *(const uint2 *) p;
    const float2 a = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.x), b = __bfloat1622float2(*(const __nv_bfloat162 *) &raw.y);
    v[0] = a.x; v[1] = a.y; v[2] = b.x; v[3] = b.y;
}
__device__ __forceinline__ void store4(float * p, const float (&v)[4]) { *(float4 *) p = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(bf16 * p, const float (&v)[4]) {
    uint2 o;
    *(__nv_bfloat162 *) &o.x = __floats2bfloat162_rn(v[0], v[1]);
    *(__nv_bfloat162 *) &o.y = __floats2bfloat162_rn(v[2], v[3]);
    *(uint2 *) p = o;
}

// bf16 activations: fast exponential and division, a few ulp of fp32; fp32 ones: the accurate forms.
template <typename T> __device__ __forceinline__ float sigmoid(float v);
template <> __device__ __forceinline__ float sigmoid<bf16>(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
template <> __device__ __forceinline__ float sigmoid<float>(float v) { return 1.f / (1.f + expf(-v)); }
template <typename T> __device__ __forceinline__ float silu(float g) { return g * sigmoid<T>(g); }

// ---- out[t] = h[t] + sum_j w[j] * h[t - taps + 1 + j], or silu(bias + sum_j w[j] * h[t - taps + 1 + j]) (ACT) ------------------
// A CTA takes a run of CONV_RUN tokens of one sequence (runs are counted from the sequence's first token in the batch) and a slice
// of the channels.  Up to CONV_TAPS taps only a sequence's first run reaches back to the stored rows: it loads every row once,
// slides over them in registers and then, as their only reader, replaces the stored rows by the range's last ones.  Longer
// filters go token by token; there the first token's CTA computes the first taps - 1 tokens for the same reason.
constexpr int CONV_RUN = 4, CONV_TAPS = 4, CONV_NT = 128;
static_assert(CONV_RUN >= CONV_TAPS - 1, "only the first run may reach back to the stored rows");

// Run c of the batch -> (sequence, run inside it): sequence b's runs start at index q_start[b] / CONV_RUN + b, which leaves room for
// every partial run before it; indices in the gaps have no tokens.
__device__ __forceinline__ int run_key(const int * q_start, int b) { return q_start[b] / CONV_RUN + b; }

// what the filter's sum starts from, and what becomes of it
template <bool ACT> __device__ __forceinline__ void conv_begin(const float (&x)[4], const float (&k)[4], const float (&b)[4], float (&c)[4]) {
#pragma unroll
    for (int e = 0; e < 4; ++e) c[e] = (ACT ? b[e] : x[e]) + k[e] * x[e];
}
template <typename T, bool ACT> __device__ __forceinline__ void conv_store(T * p, float (&c)[4]) {
    if (ACT) {
#pragma unroll
        for (int e = 0; e < 4; ++e) c[e] = silu<T>(c[e]);
    }
    store4(p, c);
}

template <typename T, bool ACT>
__device__ __noinline__ void conv_run_long(const T * h, long long ldh, const float * w, const float (&b)[4], int taps, T * st, bool past, bool keep,
                                           int q0, int n, int i0, int d, int ch, T * out) {
    const int n_old = taps - 1;
    for (int i = i0; i < min(n, i0 + CONV_RUN); ++i) {
        if (i > 0 && i < n_old) continue;
        for (int r = i; r < (i == 0 ? min(n, max(n_old, 1)) : i + 1); ++r) {
            float x[4], k[4], c[4];
            load4(h + (size_t) (q0 + r) * ldh + ch, x);
            load4(w + (size_t) n_old * d + ch, k);
            conv_begin<ACT>(x, k, b, c);
            for (int j = 0; j < n_old; ++j) {
                const int src = r - n_old + j;
                if (src >= 0) load4(h + (size_t) (q0 + src) * ldh + ch, x);
                else if (past) load4(st + (size_t) (src + n_old) * d, x);
                else continue;
                load4(w + (size_t) j * d + ch, k);
#pragma unroll
                for (int e = 0; e < 4; ++e) c[e] += k[e] * x[e];
            }
            conv_store<T, ACT>(out + (size_t) (q0 + r) * d + ch, c);
        }
        if (i == 0 && keep) {
            for (int j = 0; j < n_old; ++j) {              // ascending: entry j only needs old entries behind it
                const int src = n - n_old + j;
                float x[4] = {0.f, 0.f, 0.f, 0.f};
                if (src >= 0) load4(h + (size_t) (q0 + src) * ldh + ch, x);
                else if (past) load4(st + (size_t) (src + n_old) * d, x);
                store4(st + (size_t) j * d, x);
            }
        }
    }
}

template <typename T, bool ACT>
__global__ void __launch_bounds__(CONV_NT) causal_conv_kernel(const T * __restrict__ h, long long ldh, const float * __restrict__ w,
                                                              const float * __restrict__ bias, int taps, T * __restrict__ state, int n_state, const int * __restrict__ seq_slots,
                                                              const int * __restrict__ positions, const int * __restrict__ q_start,
                                                              int n_seqs, int d, T * __restrict__ out, int * status) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int b = 0, hi = n_seqs;
    while (hi - b > 1) {
        const int mid = (b + hi) >> 1;
        if (run_key(q_start, mid) <= (int) blockIdx.x) b = mid; else hi = mid;
    }
    const int q0 = q_start[b], n = q_start[b + 1] - q0, i0 = ((int) blockIdx.x - run_key(q_start, b)) * CONV_RUN;
    const int ch = 4 * (blockIdx.y * CONV_NT + threadIdx.x);
    if (i0 < 0 || i0 >= n || ch >= d) return;
    const int n_old = taps - 1;
    int slot = -1;
    bool past = false;
    if (i0 == 0) {
        slot = seq_slots[b];
        if (slot >= n_state) {
            if (threadIdx.x == 0) jib_report(status, JIB_ERR_BOUNDS, 42, slot);
            slot = -1;
        }
        past = slot >= 0 && positions[q0] > 0;
    }
    T * st = state + (size_t) (slot < 0 ? 0 : slot) * n_old * d + ch;
    float b4[4] = {0.f, 0.f, 0.f, 0.f};
    if (ACT) load4(bias + ch, b4);
    if (taps > CONV_TAPS) {
        conv_run_long<T, ACT>(h, ldh, w, b4, taps, st, past, slot >= 0, q0, n, i0, d, ch, out);
        return;
    }
    // rows i0 - (CONV_TAPS - 1) .. i0 + CONV_RUN - 1 in x; taps right-aligned in k; the range's last rows for the stored ones in z
    float x[CONV_RUN + CONV_TAPS - 1][4], k[CONV_TAPS][4], z[CONV_TAPS - 1][4];
    const T * hb = h + (size_t) q0 * ldh + ch;
#pragma unroll
    for (int r = 0; r < CONV_RUN + CONV_TAPS - 1; ++r) {
        const int i = i0 + r - (CONV_TAPS - 1);
#pragma unroll
        for (int e = 0; e < 4; ++e) x[r][e] = 0.f;
        if (r >= CONV_TAPS - taps && i < n) {
            if (i >= 0) load4(hb + (size_t) i * ldh, x[r]);
            else if (past) load4(st + (size_t) (i + n_old) * d, x[r]);
        }
    }
#pragma unroll
    for (int j = 0; j < CONV_TAPS; ++j)
        if (j >= CONV_TAPS - taps) load4(w + (size_t) (j - (CONV_TAPS - taps)) * d + ch, k[j]);
    if (slot >= 0) {
#pragma unroll
        for (int j = 0; j < CONV_TAPS - 1; ++j) {
            const int i = n - n_old + j;                     // negative: an old row moves up
#pragma unroll
            for (int e = 0; e < 4; ++e) z[j][e] = 0.f;
            if (j < n_old) {
                if (i >= 0) load4(hb + (size_t) i * ldh, z[j]);
                else if (past) load4(st + (size_t) (i + n_old) * d, z[j]);
            }
        }
    }
#pragma unroll
    for (int r = 0; r < CONV_RUN; ++r) {
        if (i0 + r >= n) break;
        float c[4];
        conv_begin<ACT>(x[r + CONV_TAPS - 1], k[CONV_TAPS - 1], b4, c);
#pragma unroll
        for (int j = 0; j < CONV_TAPS - 1; ++j)
            if (j >= CONV_TAPS - taps)
#pragma unroll
                for (int e = 0; e < 4; ++e) c[e] += k[j][e] * x[r + j][e];
        conv_store<T, ACT>(out + (size_t) (q0 + i0 + r) * d + ch, c);
    }
    if (slot >= 0) {
#pragma unroll
        for (int j = 0; j < CONV_TAPS - 1; ++j)
            if (j < n_old) store4(st + (size_t) j * d, z[j]);
    }
}

// ---- minGRU: S_t = (1 - z_t) S_(t-1) + z_t c_t,  y_t = S_t * silu(g_t) -------------------------------------------------------
// zxg [T][ld]: pre-activations of z, of the candidate and of the output gate, W columns each.  All arithmetic fp32.
template <typename T> __device__ __forceinline__ void gru_terms(float az, float au, float & a, float & b) {
    const float z = sigmoid<T>(az), c = sigmoid<T>(au);
    a = 1.f - z;
    b = z * (au >= 0.f ? au + 0.5f : c);
}
// Two adjacent elements at p.  PAIR: one access; else two, the second at p + step (0 at the last channel: no branch around a load,
// so that a round's loads are all in flight together).
template <bool PAIR> __device__ __forceinline__ float2 load2(const bf16 * p, int step) {
    if (PAIR) return __bfloat1622float2(*(const __nv_bfloat162 *) p);
    return make_float2(__bfloat162float(p[0]), __bfloat162float(p[step]));
}
template <bool PAIR> __device__ __forceinline__ float2 load2(const float * p, int step) {
    if (PAIR) return *(const float2 *) p;
    return make_float2(p[0], p[step]);
}
template <bool PAIR> __device__ __forceinline__ void store2(bf16 * p, float a, float b, int step) {
    if (PAIR) {
        *(__nv_bfloat162 *) p = __floats2bfloat162_rn(a, b);
    } else {
        put(p, a);
        if (step) put(p + 1, b);
    }
}
template <bool PAIR> __device__ __forceinline__ void store2(float * p, float a, float b, int step) {
    if (PAIR) {
        *(float2 *) p = make_float2(a, b);
    } else {
        put(p, a);
        if (step) put(p + 1, b);
    }
}

// One token per sequence (decode): grid (ceil(W / 256), T), row t belongs to sequence t.
template <typename T>
__global__ void __launch_bounds__(256) mingru_step_kernel(const T * __restrict__ zxg, long long ld, const float * __restrict__ zb,
                                                          const float * __restrict__ xb, float * __restrict__ state, int n_state,
                                                          const int * __restrict__ seq_slots, const int * __restrict__ positions, int W,
                                                          T * __restrict__ y, int * status) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int t = blockIdx.y, ch = blockIdx.x * 256 + threadIdx.x;
    if (ch >= W) return;
    int slot = seq_slots[t];
    if (slot >= n_state) {
        if (ch == 0) jib_report(status, JIB_ERR_BOUNDS, 43, slot);
        slot = -1;
    }
    const T * row = zxg + (size_t) t * ld;
    float * st = state + (size_t) (slot < 0 ? 0 : slot) * W + ch;
    float a, b;
    gru_terms<T>(to_f(row[ch]) + zb[ch], to_f(row[W + ch]) + xb[ch], a, b);
    const float s = (slot >= 0 && positions[t] > 0) ? a * *st + b : b;
    if (slot >= 0) *st = s;
    put(y + (size_t) t * W + ch, s * silu<T>(to_f(row[2 * W + ch])));
}

// Ranges of any length: grid (ceil(W / 16), n_seqs, 8), 256 threads = 8 channel pairs x 32 runs of SCAN_L tokens; the 8 CTAs of a
// (channel tile, sequence) form a thread-block cluster over consecutive time chunks.  Every thread composes its run
// (S -> A S + B), the runs are scanned across the warp and the CTA, the chunks' compositions are exchanged through distributed
// shared memory, and each thread replays its run from the value that gives it: every input is read once,
// SCAN_CHUNK * SCAN_CTAS tokens per round.  A range of one chunk involves the first CTA only.
constexpr int SCAN_L = 4, SCAN_CH = 16, SCAN_RUNS = 32, SCAN_CTAS = 8, SCAN_CHUNK = SCAN_L * SCAN_RUNS, SCAN_NT = 8 * SCAN_RUNS;

__device__ __forceinline__ void cluster_arrive() { asm volatile("barrier.cluster.arrive.release;" ::: "memory"); }
__device__ __forceinline__ void cluster_wait() { asm volatile("barrier.cluster.wait.acquire;" ::: "memory"); }
__device__ __forceinline__ float2 ld_cluster(const float2 * p, int rank) {
    uint32_t remote;
    float2 v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(remote) : "r"((uint32_t) __cvta_generic_to_shared(p)), "r"(rank));
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(remote) : "memory");
    return v;
}

template <typename T, bool PAIR>
__global__ void __launch_bounds__(SCAN_NT, 4) mingru_scan_kernel(const T * __restrict__ zxg, long long ld, const float * __restrict__ zb,
                                                                 const float * __restrict__ xb, float * __restrict__ state, int n_state,
                                                                 const int * __restrict__ seq_slots, const int * __restrict__ positions,
                                                                 const int * __restrict__ q_start, int W, T * __restrict__ y, int * status) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    __shared__ float2 wc[SCAN_CH][SCAN_NT / 32 + 1];         // composition of each warp's four runs, then of the warps before it
    __shared__ float2 total[SCAN_CH];                        // composition of this CTA's chunk, read by the cluster
    __shared__ float s_in[SCAN_CH];                          // state before this CTA's chunk
    const int b = blockIdx.y, q0 = q_start[b], n = q_start[b + 1] - q0, rank = blockIdx.z;
    const bool alone = n <= SCAN_CHUNK;                      // the same for all CTAs of the cluster
    if (n <= 0 || (alone && rank != 0)) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cp = threadIdx.x & 7, run = threadIdx.x >> 3;
    const int ch = blockIdx.x * SCAN_CH + 2 * cp;
    int slot = seq_slots[b];
    if (slot >= n_state) {
        if (threadIdx.x == 0 && blockIdx.x == 0) jib_report(status, JIB_ERR_BOUNDS, 44, slot);
        slot = -1;
    }
    float carry = 0.f;                                       // threads 0 .. 15: their channel's state before the round (first used after
    if (threadIdx.x < SCAN_CH) {                             // the round's own loads have been requested)
        const int c = blockIdx.x * SCAN_CH + threadIdx.x;
        if (slot >= 0 && positions[q0] > 0 && c < W) carry = state[(size_t) slot * W + c];
    }
    const bool mine = ch < W;
    const int step = ch + 1 < W ? 1 : 0, chc = min(ch, W - 1 - (PAIR ? 1 : 0));      // an idle thread reads what another one owns
    const float bz[2] = {zb[chc], zb[chc + step]}, bx[2] = {xb[chc], xb[chc + step]};
    const T * const base = zxg + (size_t) q0 * ld + chc;
    for (int t0 = rank * SCAN_CHUNK; t0 - rank * SCAN_CHUNK < n; t0 += SCAN_CHUNK * SCAN_CTAS) {
        float a[SCAN_L][2], v[SCAN_L][2];
        float2 g[SCAN_L];
        float A[2] = {1.f, 1.f}, B[2] = {0.f, 0.f};
#pragma unroll
        for (int l = 0; l < SCAN_L; ++l) {                             // every load of the round first
            const T * row = base + (size_t) min(t0 + run * SCAN_L + l, n - 1) * ld;
            const float2 az = load2<PAIR>(row, step), au = load2<PAIR>(row + W, step);
            g[l] = load2<PAIR>(row + 2 * W, step);
            a[l][0] = az.x; a[l][1] = az.y; v[l][0] = au.x; v[l][1] = au.y;
        }
#pragma unroll
        for (int l = 0; l < SCAN_L; ++l) {
            const bool live = t0 + run * SCAN_L + l < n;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                float ta, tv;
                gru_terms<T>(a[l][e] + bz[e], v[l][e] + bx[e], ta, tv);
                a[l][e] = live ? ta : 1.f;                              // past the end: S passes through
                v[l][e] = live ? tv : 0.f;
                B[e] = a[l][e] * B[e] + v[l][e];
                A[e] *= a[l][e];
            }
        }
        // the four runs of this warp: lanes 8 apart hold consecutive runs of the same channels
        float xa[2], xv[2];                                             // exclusive: the runs before mine inside the warp
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            float ia = A[e], ib = B[e];
#pragma unroll
            for (int o = 8; o < 32; o <<= 1) {
                const float pa = __shfl_up_sync(0xffffffffu, ia, o), pb = __shfl_up_sync(0xffffffffu, ib, o);
                if (lane >= o) { ib = ia * pb + ib; ia *= pa; }
            }
            if (lane >= 24) wc[2 * cp + e][warp] = make_float2(ia, ib);
            xa[e] = __shfl_up_sync(0xffffffffu, ia, 8);
            xv[e] = __shfl_up_sync(0xffffffffu, ib, 8);
            if (lane < 8) { xa[e] = 1.f; xv[e] = 0.f; }
        }
        __syncthreads();
        if (threadIdx.x < SCAN_CH * 8) {                                // 8 lanes scan the 8 warps' compositions of one channel
            const int c = threadIdx.x >> 3, k = threadIdx.x & 7;
            float ia = wc[c][k].x, ib = wc[c][k].y;
#pragma unroll
            for (int o = 1; o < 8; o <<= 1) {
                const float pa = __shfl_up_sync(0xffffffffu, ia, o, 8), pb = __shfl_up_sync(0xffffffffu, ib, o, 8);
                if (k >= o) { ib = ia * pb + ib; ia *= pa; }
            }
            float ea = __shfl_up_sync(0xffffffffu, ia, 1, 8), eb = __shfl_up_sync(0xffffffffu, ib, 1, 8);
            if (k == 0) { ea = 1.f; eb = 0.f; }
            wc[c][k] = make_float2(ea, eb);
            if (k == 7) total[c] = make_float2(ia, ib);
        }
        if (alone) {
            __syncthreads();
        } else {
            cluster_arrive();
            cluster_wait();
        }
        if (threadIdx.x < SCAN_CH) {
            float s = carry;
            if (alone) {
                s_in[threadIdx.x] = s;
                s = total[threadIdx.x].x * s + total[threadIdx.x].y;
            } else {
                float2 m[SCAN_CTAS];
#pragma unroll
                for (int r = 0; r < SCAN_CTAS; ++r) m[r] = ld_cluster(&total[threadIdx.x], r);
#pragma unroll
                for (int r = 0; r < SCAN_CTAS; ++r) {
                    if (r == rank) s_in[threadIdx.x] = s;
                    s = m[r].x * s + m[r].y;
                }
            }
            carry = s;
        }
        __syncthreads();
        if (!alone) cluster_arrive();        // this CTA has read its peers' compositions
        {
            const float2 w0 = wc[2 * cp][warp], w1 = wc[2 * cp + 1][warp];
            float s0 = xa[0] * (w0.x * s_in[2 * cp] + w0.y) + xv[0], s1 = xa[1] * (w1.x * s_in[2 * cp + 1] + w1.y) + xv[1];
#pragma unroll
            for (int l = 0; l < SCAN_L; ++l) {
                const int t = t0 + run * SCAN_L + l;
                s0 = a[l][0] * s0 + v[l][0];
                s1 = a[l][1] * s1 + v[l][1];
                const float y0 = s0 * silu<T>(g[l].x), y1 = s1 * silu<T>(g[l].y);
                if (t < n && mine) store2<PAIR>(y + (size_t) (q0 + t) * W + ch, y0, y1, step);
            }
        }
        // the compositions are rewritten in the next round, and a CTA that leaves takes its shared memory with it
        if (!alone) cluster_wait();
    }
    if (threadIdx.x < SCAN_CH && slot >= 0 && rank == 0) {
        const int c = blockIdx.x * SCAN_CH + threadIdx.x;
        if (c < W) state[(size_t) slot * W + c] = carry;
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

}  // namespace

extern "C" {

JIB_EXPORT int jib_causal_conv(const void * h, long long ldh, const float * w, const float * bias, int silu, int taps, void * state, int n_state,
                               const int * seq_slots, const int * positions, const int * q_start, int n_seqs, int T, int d, int f32, void * out,
                               int * status, void * stream) {
    if (T <= 0 || n_seqs <= 0) return 0;
    if (d % 4 || ldh % 4 || taps < 1 || (taps > 1 && state == nullptr) || (silu && bias == nullptr)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    const dim3 grid(T / CONV_RUN + n_seqs, (d / 4 + CONV_NT - 1) / CONV_NT);
#define CALL(TT, ACT)                                                                                                                       \
    JIB_LAUNCH((causal_conv_kernel<TT, ACT>), grid, CONV_NT, 0, s, (const TT *) h, ldh, w, bias, taps, (TT *) state, n_state, seq_slots, positions, \
               q_start, n_seqs, d, (TT *) out, status)
    if (f32) {
        if (silu) CALL(float, true);
        else CALL(float, false);
    } else {
        if (silu) CALL(bf16, true);
        else CALL(bf16, false);
    }
#undef CALL
    return launched();
}

JIB_EXPORT int jib_mingru(const void * zxg, long long ld, const float * zb, const float * xb, float * state, int n_state,
                          const int * seq_slots, const int * positions, const int * q_start, int n_seqs, int T, int W, int single, int f32,
                          void * y, int * status, void * stream) {
    if (T <= 0 || n_seqs <= 0) return 0;
    if (W < 1 || ld < 3LL * W || n_seqs > 65535 || T > 2147483647 / 4) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    if (single) {
        if (T > 65535) return JIB_E_ARG;
        const dim3 grid((W + 255) / 256, T);
        if (f32)
            JIB_LAUNCH((mingru_step_kernel<float>), grid, 256, 0, s, (const float *) zxg, ld, zb, xb, state, n_state, seq_slots, positions, W,
                       (float *) y, status);
        else
            JIB_LAUNCH((mingru_step_kernel<bf16>), grid, 256, 0, s, (const bf16 *) zxg, ld, zb, xb, state, n_state, seq_slots, positions, W,
                       (bf16 *) y, status);
    } else {
        const dim3 grid((W + SCAN_CH - 1) / SCAN_CH, n_seqs, SCAN_CTAS);
        const size_t el = f32 ? 4 : 2;
        const bool pair = W % 2 == 0 && ld % 2 == 0 && (((uintptr_t) zxg | (uintptr_t) y) & (2 * el - 1)) == 0;
        cudaError_t e;
#define JIB_SCAN(TT, PAIR)                                                                                                            \
    e = jib::launch_pdl_cluster(mingru_scan_kernel<TT, PAIR>, grid, dim3(SCAN_NT), 0, s, SCAN_CTAS, (const TT *) zxg, ld, zb, xb, state, \
                                n_state, seq_slots, positions, q_start, W, (TT *) y, status)
        if (f32) {
            if (pair) JIB_SCAN(float, true);
            else JIB_SCAN(float, false);
        } else {
            if (pair) JIB_SCAN(bf16, true);
            else JIB_SCAN(bf16, false);
        }
#undef JIB_SCAN
        if (e != cudaSuccess) { (void) cudaGetLastError(); return JIB_E_LAUNCH; }
    }
    return launched();
}

}  // extern "C"
