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

__device__ __forceinline__ int find_seq(const int * q_start, int n_seqs, int t) {
    int lo = 0, hi = n_seqs;
    while (hi - lo > 1) {
        const int mid = (lo + hi) >> 1;
        if (q_start[mid] <= t) lo = mid; else hi = mid;
    }
    return lo;
}

// ---- out[t] = h[t] + sum_j w[j] * h[t - taps + 1 + j] --------------------------------------------------------------------
// grid (ceil(T / CONV_RUN)): a CTA takes a run of tokens.  A run inside one sequence and past its first taps - 1 tokens loads every
// row once and slides over them in registers.  The first taps - 1 tokens of a sequence's range read the stored rows, so one CTA
// (the first token's) computes all of them and then, as the only reader, writes the stored rows of the range's end.
constexpr int CONV_RUN = 4, CONV_TAPS = 4;

template <typename T>
__device__ __forceinline__ void causal_conv_token(const T * __restrict__ h, const float * __restrict__ w, int taps, T * __restrict__ state,
                                                  int n_state, const int * __restrict__ seq_slots, const int * __restrict__ positions,
                                                  const int * __restrict__ q_start, int n_seqs, int d, T * __restrict__ out, int * status,
                                                  int t);

template <typename T>
__global__ void __launch_bounds__(256) causal_conv_kernel(const T * __restrict__ h, const float * __restrict__ w, int taps,
                                                          T * __restrict__ state, int n_state, const int * __restrict__ seq_slots,
                                                          const int * __restrict__ positions, const int * __restrict__ q_start, int n_seqs,
                                                          int n_tok, int d, T * __restrict__ out, int * status) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int t0 = blockIdx.x * CONV_RUN, t1 = min(n_tok, t0 + CONV_RUN);
    const int b = find_seq(q_start, n_seqs, t0);
    const bool inner = taps <= CONV_TAPS && t0 - q_start[b] >= taps - 1 && t0 + CONV_RUN <= q_start[b + 1];
    if (!inner) {
        for (int t = t0; t < t1; ++t)
            causal_conv_token(h, w, taps, state, n_state, seq_slots, positions, q_start, n_seqs, d, out, status, t);
        return;
    }
    const int n_old = taps - 1;
    for (int v = threadIdx.x; v < d / 4; v += blockDim.x) {
        const int ch = 4 * v;
        float x[CONV_RUN + CONV_TAPS - 1][4], k[CONV_TAPS][4];        // rows t0 - CONV_TAPS + 1 .. ; taps, the last one in k[CONV_TAPS - 1]
#pragma unroll
        for (int r = 0; r < CONV_RUN + CONV_TAPS - 1; ++r)
            if (r >= CONV_TAPS - 1 - n_old) load4(h + (size_t) (t0 + r - (CONV_TAPS - 1)) * d + ch, x[r]);
#pragma unroll
        for (int j = 0; j < CONV_TAPS; ++j)
            if (j >= CONV_TAPS - taps) load4(w + (size_t) (j - (CONV_TAPS - taps)) * d + ch, k[j]);
#pragma unroll
        for (int r = 0; r < CONV_RUN; ++r) {
            float c[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) c[e] = x[r + CONV_TAPS - 1][e] + k[CONV_TAPS - 1][e] * x[r + CONV_TAPS - 1][e];
#pragma unroll
            for (int j = 0; j < CONV_TAPS - 1; ++j)
                if (j >= CONV_TAPS - taps)
#pragma unroll
                    for (int e = 0; e < 4; ++e) c[e] += k[j][e] * x[r + j][e];
            store4(out + (size_t) (t0 + r) * d + ch, c);
        }
    }
}

template <typename T>
__device__ __forceinline__ void causal_conv_token(const T * __restrict__ h, const float * __restrict__ w, int taps, T * __restrict__ state,
                                                  int n_state, const int * __restrict__ seq_slots, const int * __restrict__ positions,
                                                  const int * __restrict__ q_start, int n_seqs, int d, T * __restrict__ out, int * status,
                                                  int t) {
    const int b = find_seq(q_start, n_seqs, t);
    const int q0 = q_start[b], n = q_start[b + 1] - q0, i = t - q0;
    if (i < 0 || i >= n || (i > 0 && i < taps - 1)) return;
    const int n_old = taps - 1;
    int slot = -1;
    bool past = false;
    if (i == 0) {
        slot = seq_slots[b];
        if (slot >= n_state) {
            if (threadIdx.x == 0) jib_report(status, JIB_ERR_BOUNDS, 42, slot);
            slot = -1;
        }
        past = slot >= 0 && positions[q0] > 0;
    }
    const int i_end = i == 0 ? min(n, max(n_old, 1)) : i + 1;
    for (int v = threadIdx.x; v < d / 4; v += blockDim.x) {
        const int ch = 4 * v;
        T * st = state + (size_t) (slot < 0 ? 0 : slot) * n_old * d + ch;
        for (int r = i; r < i_end; ++r) {
            float x[4], k[4], c[4];
            load4(h + (size_t) (q0 + r) * d + ch, x);
            load4(w + (size_t) n_old * d + ch, k);
#pragma unroll
            for (int e = 0; e < 4; ++e) c[e] = x[e] + k[e] * x[e];
            for (int j = 0; j < n_old; ++j) {
                const int src = r - n_old + j;
                if (src >= 0) load4(h + (size_t) (q0 + src) * d + ch, x);
                else if (past) load4(st + (size_t) (src + n_old) * d, x);
                else continue;
                load4(w + (size_t) j * d + ch, k);
#pragma unroll
                for (int e = 0; e < 4; ++e) c[e] += k[e] * x[e];
            }
            store4(out + (size_t) (q0 + r) * d + ch, c);
        }
        if (i == 0 && slot >= 0) {
            for (int j = 0; j < n_old; ++j) {              // ascending: entry j only needs old entries behind it
                const int src = n - n_old + j;
                float x[4] = {0.f, 0.f, 0.f, 0.f};
                if (src >= 0) load4(h + (size_t) (q0 + src) * d + ch, x);
                else if (past) load4(st + (size_t) (src + n_old) * d, x);
                store4(st + (size_t) j * d, x);
            }
        }
    }
}

// ---- minGRU: S_t = (1 - z_t) S_(t-1) + z_t c_t,  y_t = S_t * silu(g_t) -------------------------------------------------------
// zxg [T][ld]: pre-activations of z, of the candidate and of the output gate, W columns each.  All arithmetic fp32.
// (bf16 activations: fast exponential and division, a few ulp of fp32; fp32 ones: the accurate forms)
template <typename T> __device__ __forceinline__ float sigmoid(float v);
template <> __device__ __forceinline__ float sigmoid<bf16>(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
template <> __device__ __forceinline__ float sigmoid<float>(float v) { return 1.f / (1.f + expf(-v)); }
template <typename T> __device__ __forceinline__ void gru_terms(float az, float au, float & a, float & b) {
    const float z = sigmoid<T>(az), c = sigmoid<T>(au);
    a = 1.f - z;
    b = z * (au >= 0.f ? au + 0.5f : c);
}
template <typename T> __device__ __forceinline__ float silu(float g) { return g * sigmoid<T>(g); }
// Two adjacent elements; pair: the address is a multiple of their size (else, or past the last channel, one by one).
__device__ __forceinline__ float2 load2(const bf16 * p, bool pair, bool second) {
    if (pair) return __bfloat1622float2(*(const __nv_bfloat162 *) p);
    return make_float2(__bfloat162float(p[0]), second ? __bfloat162float(p[1]) : 0.f);
}
__device__ __forceinline__ float2 load2(const float * p, bool pair, bool second) {
    if (pair) return *(const float2 *) p;
    return make_float2(p[0], second ? p[1] : 0.f);
}
__device__ __forceinline__ void store2(bf16 * p, float a, float b, bool pair, bool second) {
    if (pair) *(__nv_bfloat162 *) p = __floats2bfloat162_rn(a, b);
    else { put(p, a); if (second) put(p + 1, b); }
}
__device__ __forceinline__ void store2(float * p, float a, float b, bool pair, bool second) {
    if (pair) *(float2 *) p = make_float2(a, b);
    else { put(p, a); if (second) put(p + 1, b); }
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

// Ranges of any length: grid (ceil(W / 16), n_seqs), 1024 threads = 8 channel pairs x 128 runs of SCAN_L tokens.  Every thread
// composes its run (S -> A S + B), the runs are scanned across the CTA, and each thread replays its run from the value the
// scan gives it: every input is read once, SCAN_L * 128 tokens per round, the carry between rounds stays in shared memory.
constexpr int SCAN_L = 4, SCAN_CH = 16, SCAN_RUNS = 128;
template <typename T>
__global__ void __launch_bounds__(1024) mingru_scan_kernel(const T * __restrict__ zxg, long long ld, const float * __restrict__ zb,
                                                           const float * __restrict__ xb, float * __restrict__ state, int n_state,
                                                           const int * __restrict__ seq_slots, const int * __restrict__ positions,
                                                           const int * __restrict__ q_start, int W, T * __restrict__ y, int * status) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    __shared__ float wa[SCAN_CH][33], wb[SCAN_CH][33];       // per warp: composition of its four runs, then of the warps before it
    __shared__ float carry[SCAN_CH];
    const int b = blockIdx.y, q0 = q_start[b], n = q_start[b + 1] - q0;
    if (n <= 0) return;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int cp = threadIdx.x & 7, run = threadIdx.x >> 3;
    const int ch = blockIdx.x * SCAN_CH + 2 * cp;
    int slot = seq_slots[b];
    if (slot >= n_state) {
        if (threadIdx.x == 0 && blockIdx.x == 0) jib_report(status, JIB_ERR_BOUNDS, 44, slot);
        slot = -1;
    }
    if (threadIdx.x < SCAN_CH) {
        const int c = blockIdx.x * SCAN_CH + threadIdx.x;
        carry[threadIdx.x] = (slot >= 0 && positions[q0] > 0 && c < W) ? state[(size_t) slot * W + c] : 0.f;
    }
    const bool in[2] = {ch < W, ch + 1 < W};
    const bool pair = (W & 1) == 0 && (ld & 1) == 0 && (((uintptr_t) zxg | (uintptr_t) y) & (2 * sizeof(T) - 1)) == 0;
    const float bz[2] = {in[0] ? zb[ch] : 0.f, in[1] ? zb[ch + 1] : 0.f};
    const float bx[2] = {in[0] ? xb[ch] : 0.f, in[1] ? xb[ch + 1] : 0.f};
    __syncthreads();
    for (int t0 = 0; t0 < n; t0 += SCAN_L * SCAN_RUNS) {
        float a[SCAN_L][2], v[SCAN_L][2];
        float2 g[SCAN_L];
        float A[2] = {1.f, 1.f}, B[2] = {0.f, 0.f};
#pragma unroll
        for (int l = 0; l < SCAN_L; ++l) {                             // every load of the round first
            const int t = t0 + run * SCAN_L + l;
            const T * row = zxg + (size_t) (q0 + t) * ld + ch;
            float2 az = make_float2(0.f, 0.f), au = az;
            g[l] = az;
            if (t < n && in[0]) {
                az = load2(row, pair, in[1]);
                au = load2(row + W, pair, in[1]);
                g[l] = load2(row + 2 * W, pair, in[1]);
            }
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
            if (lane >= 24) { wa[2 * cp + e][warp] = ia; wb[2 * cp + e][warp] = ib; }
            xa[e] = __shfl_up_sync(0xffffffffu, ia, 8);
            xv[e] = __shfl_up_sync(0xffffffffu, ib, 8);
            if (lane < 8) { xa[e] = 1.f; xv[e] = 0.f; }
        }
        __syncthreads();
        if (warp < SCAN_CH) {                                           // warp c scans the 32 warps' compositions of channel c
            const float s0 = carry[warp];
            float ia = wa[warp][lane], ib = wb[warp][lane];
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float pa = __shfl_up_sync(0xffffffffu, ia, o), pb = __shfl_up_sync(0xffffffffu, ib, o);
                if (lane >= o) { ib = ia * pb + ib; ia *= pa; }
            }
            const float s_end = ia * s0 + ib;                           // state after warp `lane`'s runs
            float s_in = __shfl_up_sync(0xffffffffu, s_end, 1);
            if (lane == 0) s_in = s0;
            __syncwarp();
            wa[warp][lane] = s_in;                                      // state before warp `lane`'s runs
            if (lane == 31) carry[warp] = s_end;
        }
        __syncthreads();
        {
            float s0 = xa[0] * wa[2 * cp][warp] + xv[0], s1 = xa[1] * wa[2 * cp + 1][warp] + xv[1];
#pragma unroll
            for (int l = 0; l < SCAN_L; ++l) {
                const int t = t0 + run * SCAN_L + l;
                s0 = a[l][0] * s0 + v[l][0];
                s1 = a[l][1] * s1 + v[l][1];
                if (t < n && in[0])
                    store2(y + (size_t) (q0 + t) * W + ch, s0 * silu<T>(g[l].x), s1 * silu<T>(g[l].y), pair, in[1]);
            }
        }
        __syncthreads();                                                // wa / wb are rewritten in the next round
    }
    if (threadIdx.x < SCAN_CH && slot >= 0) {
        const int c = blockIdx.x * SCAN_CH + threadIdx.x;
        if (c < W) state[(size_t) slot * W + c] = carry[threadIdx.x];
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

}  // namespace

extern "C" {

JIB_EXPORT int jib_causal_conv(const void * h, const float * w, int taps, void * state, int n_state, const int * seq_slots,
                               const int * positions, const int * q_start, int n_seqs, int T, int d, int f32, void * out, int * status,
                               void * stream) {
    if (T <= 0 || n_seqs <= 0) return 0;
    if (d % 4 || taps < 1 || (taps > 1 && state == nullptr)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    const int grid = (T + CONV_RUN - 1) / CONV_RUN;
    if (f32)
        JIB_LAUNCH((causal_conv_kernel<float>), grid, 256, 0, s, (const float *) h, w, taps, (float *) state, n_state, seq_slots, positions,
                   q_start, n_seqs, T, d, (float *) out, status);
    else
        JIB_LAUNCH((causal_conv_kernel<bf16>), grid, 256, 0, s, (const bf16 *) h, w, taps, (bf16 *) state, n_state, seq_slots, positions,
                   q_start, n_seqs, T, d, (bf16 *) out, status);
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
        const dim3 grid((W + SCAN_CH - 1) / SCAN_CH, n_seqs);
        if (f32)
            JIB_LAUNCH((mingru_scan_kernel<float>), grid, 1024, 0, s, (const float *) zxg, ld, zb, xb, state, n_state, seq_slots, positions,
                       q_start, W, (float *) y, status);
        else
            JIB_LAUNCH((mingru_scan_kernel<bf16>), grid, 1024, 0, s, (const bf16 *) zxg, ld, zb, xb, state, n_state, seq_slots, positions,
                       q_start, W, (bf16 *) y, status);
    }
    return launched();
}

}  // extern "C"
