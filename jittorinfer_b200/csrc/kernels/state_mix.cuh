// Device helpers shared by the matrix-state mixers (state_mix.cu, state_chunk.cu).
#pragma once
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "sm100.cuh"

// state_chunk.cu: whether the tensor-core form covers the mixer's sizes; its three launches in place of state_prep and state_scan.
bool jib_state_chunk_ok(const jib_state_mix & a);
int jib_state_chunk_run(const jib_state_mix & a, cudaStream_t s);

namespace state_mix {

typedef __nv_bfloat16 bf16;
enum { DELTA = JIB_STATE_DELTA, LINEAR = JIB_STATE_LINEAR, SSD = JIB_STATE_SSD, HGRN = JIB_STATE_HGRN, MLSTM = JIB_STATE_MLSTM };
__host__ __device__ constexpr bool per_channel(int kind) { return kind == DELTA || kind == LINEAR || kind == HGRN; }      // decays per key channel

// Columns of the rows of v and o between the launches of a portion: MLSTM has one more, what the keys add up to (v = 1), padded to whole
// vectors of 4.
__host__ __device__ constexpr int scratch_cols(int kind, int V) { return kind == MLSTM ? (V + 4) / 4 * 4 : V; }

__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ void put(bf16 * p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void put(float * p, float v) { *p = v; }
__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// bf16 activations: fast exponential and division for gates and silu (a few ulp of fp32); fp32 ones: the accurate forms.
template <typename T> __device__ __forceinline__ float sigmoid(float v);
template <> __device__ __forceinline__ float sigmoid<bf16>(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
template <> __device__ __forceinline__ float sigmoid<float>(float v) { return 1.f / (1.f + expf(-v)); }
template <typename T> __device__ __forceinline__ float silu(float v) { return v * sigmoid<T>(v); }
__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

template <int KIND> __device__ __forceinline__ float channel_decay(const jib_state_mix & a, float z, int h) {
    return KIND == DELTA ? expf(a.neg_a[h] * softplus(z)) : expf(-a.inv_tau * softplus(-z));
}
// HGRN: decay f = l + (1 - l) sigmoid(z) and 1 - f, both without cancellation
__device__ __forceinline__ void bounded_gate(float z, float l, float & f, float & rest) {
    const float e = expf(-fabsf(z)), s = 1.f / (1.f + e), big = (1.f - l) * s, small = (1.f - l) * (e * s);      // sigmoid(|z|), sigmoid(-|z|)
    f = l + (z >= 0.f ? big : small);
    rest = z >= 0.f ? small : big;
}
// MLSTM: log gates from pre-activations
__device__ __forceinline__ float log_input_gate(float z, float cap) { return cap * tanhf(z / cap); }
__device__ __forceinline__ float log_forget_gate(float z, float cap) { return -softplus(-cap * tanhf(z / cap)); }

template <int KIND> __device__ __forceinline__ float head_factor(const jib_state_mix & a, float z, int h) {
    return KIND == DELTA ? 1.f / (1.f + expf(-z)) : softplus(z + a.bias[h]);
}

__device__ __forceinline__ int seq_of(const int * q_start, int n_seqs, int t) {
    int b = 0, hi = n_seqs;
    while (hi - b > 1) {
        const int mid = (b + hi) >> 1;
        if (q_start[mid] <= t) b = mid; else hi = mid;
    }
    return b;
}
__device__ __forceinline__ int checked_slot(const jib_state_mix & a, int b, int site) {
    const int slot = a.seq_slots[b];
    if (slot >= a.n_state) {
        if (threadIdx.x == 0) jib_report(a.status, JIB_ERR_BOUNDS, site, slot);
        return -1;
    }
    return slot;
}

// Column c of token row t (position p, back rows of its range precede it in the batch): convolved and silu'd if c lies in the window.
template <typename T>
__device__ __forceinline__ float column(const jib_state_mix & a, int t, int c, int p, int back, int slot) {
    const T * x = (const T *) a.proj + (size_t) t * a.ld + c;
    if (a.taps == 0) return to_f(*x);
    const int w = c - a.conv0;
    float acc = a.conv_b != nullptr ? a.conv_b[w] : 0.f;
    for (int j = 0; j < a.taps; ++j) {
        const int d = a.taps - 1 - j;                        // tokens back
        if (d > p) continue;
        float v;
        if (d <= back) v = to_f(x[-(long long) d * a.ld]);
        else if (slot >= 0) v = to_f(((const T *) a.conv_state)[((size_t) slot * a.taps + (p - d) % a.taps) * a.n_conv + w]);
        else continue;
        acc += a.conv_w[(size_t) j * a.n_conv + w] * v;
    }
    return silu<T>(acc);
}

// The same for a single token (nothing of its sequence precedes it in the batch): up to 4 taps all loads are in flight together.
template <typename T>
__device__ __forceinline__ float column_single(const jib_state_mix & a, int t, int c, int p, int slot) {
    if (a.taps > 4) return column<T>(a, t, c, p, 0, slot);
    const float x = to_f(((const T *) a.proj)[(size_t) t * a.ld + c]);
    if (a.taps == 0) return x;
    const int w = c - a.conv0;
    const T * ring = (const T *) a.conv_state + (size_t) (slot < 0 ? 0 : slot) * a.taps * a.n_conv + w;
    float v[3], k[4];
    int row = p % a.taps;
#pragma unroll
    for (int d = 1; d < 4; ++d) {                            // d tokens back
        row = row == 0 ? a.taps - 1 : row - 1;
        const bool in = d < a.taps && d <= p && slot >= 0;
        v[d - 1] = in ? to_f(ring[(size_t) row * a.n_conv]) : 0.f;
        k[d] = d < a.taps ? a.conv_w[(size_t) (a.taps - 1 - d) * a.n_conv + w] : 0.f;
    }
    k[0] = a.conv_w[(size_t) (a.taps - 1) * a.n_conv + w];
    const float b = a.conv_b != nullptr ? a.conv_b[w] : 0.f;
    return silu<T>(b + k[0] * x + k[1] * v[0] + k[2] * v[1] + k[3] * v[2]);
}

__device__ __forceinline__ void cp16(void * dst, const void * src) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"((uint32_t) __cvta_generic_to_shared(dst)), "l"(src) : "memory");
}
__device__ __forceinline__ void cp4(void * dst, const void * src) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"((uint32_t) __cvta_generic_to_shared(dst)), "l"(src) : "memory");
}

// The range's last convolution inputs into the ring, by threads tid of nt.  In a launch after the one that read the ring's old rows.
template <typename T>
__device__ __forceinline__ void store_conv_tail(const jib_state_mix & a, int slot, int q0, int n, int tid, int nt) {
    if (a.taps < 2 || slot < 0) return;
    const int keep = min(n, a.taps - 1), p_end = a.positions[q0] + n;
    for (int i = tid; i < keep * a.n_conv; i += nt) {
        const int d = i / a.n_conv + 1, w = i % a.n_conv;    // d tokens before the end of the range
        ((T *) a.conv_state)[((size_t) slot * a.taps + (p_end - d) % a.taps) * a.n_conv + w] =
            ((const T *) a.proj)[(size_t) (q0 + n - d) * a.ld + a.conv0 + w];
    }
}

}  // namespace state_mix
