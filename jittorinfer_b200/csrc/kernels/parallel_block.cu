// Row kernels of blocks with an fp32 residual stream whose sublayers run side by side on one norm:
//
//   h = norm(x);   x <- x + m * (sigmoid(g1) * mixer(h) + sigmoid(g2) * ff(h))
//
//   embed_norm     x = norm(embedding row), then the first block's norm
//   block_update   the sum above -- the expert-weighted combine of the feed-forward included -- then the next block's norm
//   rms_rows       norm of selected rows (before the output head)
//
// One CTA owns one token's row and keeps it in registers, so the sum, the residual store and the norm that follows are one
// pass.  In a batch of single tokens (decode) the same launch also runs the next block's input convolution against the
// sequence's stored rows and advances them.  Activations are bf16 or fp32; the residual and all arithmetic are fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "pdl.cuh"
#include "sm100.cuh"

namespace {

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
template <int NT>
__device__ __forceinline__ float block_sum(float v, float * red) {
    v = warp_sum(v);
    const int w = threadIdx.x >> 5, l = threadIdx.x & 31;
    if (l == 0) red[w] = v;
    __syncthreads();
    float t = l < NT / 32 ? red[l] : 0.f;
    t = warp_sum(t);
    __syncthreads();
    return t;
}

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
__device__ __forceinline__ void round4(float (&)[4], const float *) {}
__device__ __forceinline__ void round4(float (&v)[4], const bf16 *) {
#pragma unroll
    for (int e = 0; e < 4; ++e) v[e] = __bfloat162float(__float2bfloat16(v[e]));
}
__device__ __forceinline__ float sigmoid(float v) { return 1.f / (1.f + expf(-v)); }

// x row -> residual store, norm, and (decode) the next block's input convolution.
template <typename T, int NT, int MAXV>
__device__ __forceinline__ void finish_row(float (&v)[MAXV][4], int t, int d, const jib_row_tail & a, float * red, bool dry) {
    const int nv = d / 4;
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            if (!dry) store4((float *) a.x_out + (size_t) t * d + 4 * i, v[it]);
#pragma unroll
            for (int e = 0; e < 4; ++e) ss += v[it][e] * v[it][e];
        }
    }
    if (a.norm_w == nullptr) return;
    ss = block_sum<NT>(ss, red);
    const float inv = rsqrtf(ss / (float) d + a.eps);
    const bool conv = a.conv_w != nullptr;
    int slot = -1;
    bool past = false;
    if (conv) {
        slot = a.seq_slots[t];
        if (slot >= a.n_state) {
            if (threadIdx.x == 0 && !dry) jib_report(a.status, JIB_ERR_BOUNDS, 41, slot);
            slot = -1;
        }
        past = slot >= 0 && a.positions[t] > 0;      // a sequence's first token starts from zeros, whatever the slot held
    }
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i >= nv) continue;
        float w[4], h[4];
        load4(a.norm_w + 4 * i, w);
#pragma unroll
        for (int e = 0; e < 4; ++e) h[e] = v[it][e] * inv * w[e];
        if (!dry) store4((T *) a.h_out + (size_t) t * d + 4 * i, h);
        if (conv) {
            round4(h, (const T *) nullptr);          // the convolution reads what a later step will read back from the state
            float c[4], k[4];
            load4(a.conv_w + (size_t) (a.taps - 1) * d + 4 * i, k);
#pragma unroll
            for (int e = 0; e < 4; ++e) c[e] = h[e] + k[e] * h[e];
            T * st = (T *) a.conv_state + ((size_t) (slot < 0 ? 0 : slot) * (a.taps - 1)) * d + 4 * i;
            for (int j = 0; j < a.taps - 1; ++j) {
                float s[4] = {0.f, 0.f, 0.f, 0.f};
                if (past) {
                    load4(st + (size_t) j * d, s);
                    load4(a.conv_w + (size_t) j * d + 4 * i, k);
#pragma unroll
                    for (int e = 0; e < 4; ++e) c[e] += k[e] * s[e];
                }
                if (slot >= 0 && !dry && j > 0) store4(st + (size_t) (j - 1) * d, s);
            }
            if (slot >= 0 && !dry && a.taps > 1) store4(st + (size_t) (a.taps - 2) * d, h);
            if (!dry) store4((T *) a.hc_out + (size_t) t * d + 4 * i, c);
        }
    }
}

template <typename T, int NT, int MAXV>
__global__ void __launch_bounds__(NT) embed_norm_kernel(const T * __restrict__ table, const int * __restrict__ ids, const float * __restrict__ w,
                                                        float eps, int d, int n_vocab, const jib_row_tail tail) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int t = blockIdx.x;
    int id = ids[t];
    if (id < 0 || id >= n_vocab) {
        if (threadIdx.x == 0) jib_report(tail.status, JIB_ERR_BOUNDS, 40, id);
        id = id < 0 ? 0 : n_vocab - 1;
    }
    const int nv = d / 4;
    float v[MAXV][4];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            load4(table + (size_t) id * d + 4 * i, v[it]);
#pragma unroll
            for (int e = 0; e < 4; ++e) ss += v[it][e] * v[it][e];
        }
    }
    ss = block_sum<NT>(ss, red);
    const float inv = rsqrtf(ss / (float) d + eps);
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            float k[4];
            load4(w + 4 * i, k);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[it][e] *= inv * k[e];
        }
    }
    finish_row<T, NT, MAXV>(v, t, d, tail, red, false);
}

struct UpdateArgs {
    const float * x;            // [T][d] residual before the block
    const void * o;             // [T][d] mixer output
    const void * gates;         // [T][>= 2d]: pre-activations of the mixer's gate, then of the feed-forward's
    const float * b1, * b2;     // [d] gate biases
    const void * y;             // expert rows in sorted order, or null: no feed-forward
    const int * dest;           // [T][k] sorted row of pair (t, j), -1: none
    const float * wts;          // [T][k]
    long long gate_stride;
    int k, d;
    float mult;
};

template <typename T, int NT, int MAXV>
__device__ __noinline__ void block_update_row(const UpdateArgs & a, const jib_row_tail & tail, float * red, bool dry) {
    const int t = blockIdx.x, d = a.d, nv = d / 4;
    float v[MAXV][4];
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i >= nv) continue;
        float o[4], g[4], b[4], sum[4];
        load4((const T *) a.o + (size_t) t * d + 4 * i, o);
        load4((const T *) a.gates + (size_t) t * a.gate_stride + 4 * i, g);
        load4(a.b1 + 4 * i, b);
#pragma unroll
        for (int e = 0; e < 4; ++e) sum[e] = sigmoid(g[e] + b[e]) * o[e];
        if (a.y != nullptr) {
            float f[4] = {0.f, 0.f, 0.f, 0.f};
            for (int j = 0; j < a.k; ++j) {
                const int row = dry ? 0 : a.dest[(size_t) t * a.k + j];
                if (row < 0) continue;
                const float w = a.wts[(size_t) t * a.k + j];
                float y[4];
                load4((const T *) a.y + (size_t) row * d + 4 * i, y);
#pragma unroll
                for (int e = 0; e < 4; ++e) f[e] += w * y[e];
            }
            load4((const T *) a.gates + (size_t) t * a.gate_stride + d + 4 * i, g);
            load4(a.b2 + 4 * i, b);
#pragma unroll
            for (int e = 0; e < 4; ++e) sum[e] += sigmoid(g[e] + b[e]) * f[e];
        }
        float x[4];
        load4(a.x + (size_t) t * d + 4 * i, x);
#pragma unroll
        for (int e = 0; e < 4; ++e) v[it][e] = x[e] + a.mult * sum[e];
    }
    finish_row<T, NT, MAXV>(v, t, d, tail, red, dry);
}

template <typename T, int NT, int MAXV>
__global__ void __launch_bounds__(NT) block_update_kernel(const UpdateArgs a, const jib_row_tail tail, int warm) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    if (warm) block_update_row<T, NT, MAXV>(a, tail, red, true);
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    block_update_row<T, NT, MAXV>(a, tail, red, false);
}

// out[i] = x[rows[i]] / rms * w
template <typename T, int NT, int MAXV>
__global__ void __launch_bounds__(NT) rms_rows_kernel(const float * __restrict__ x, const int * __restrict__ rows, const float * __restrict__ w,
                                                      float eps, int d, int n_src, T * __restrict__ out) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int r = rows != nullptr ? rows[blockIdx.x] : (int) blockIdx.x;
    r = r < 0 ? 0 : (r >= n_src ? n_src - 1 : r);
    const int nv = d / 4;
    float v[MAXV][4];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            load4(x + (size_t) r * d + 4 * i, v[it]);
#pragma unroll
            for (int e = 0; e < 4; ++e) ss += v[it][e] * v[it][e];
        }
    }
    ss = block_sum<NT>(ss, red);
    const float inv = rsqrtf(ss / (float) d + eps);
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            float k[4];
            load4(w + 4 * i, k);
#pragma unroll
            for (int e = 0; e < 4; ++e) v[it][e] *= inv * k[e];
            store4(out + (size_t) blockIdx.x * d + 4 * i, v[it]);
        }
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

inline bool tail_ok(const jib_row_tail * t, int d) {
    if (t == nullptr || t->x_out == nullptr || d % 4 || d > 16384) return false;
    if (t->norm_w != nullptr && t->h_out == nullptr) return false;
    if (t->conv_w != nullptr)
        return t->norm_w != nullptr && t->hc_out != nullptr && t->taps >= 1 && (t->taps == 1 || t->conv_state != nullptr) &&
               t->seq_slots != nullptr && t->positions != nullptr && t->n_state >= 0;
    return true;
}

}  // namespace

// (threads, 4-element vectors per thread) by row width
#define JIB_ROW_DISPATCH(d, CALL)            \
    if ((d) <= 1024) CALL(256, 1);           \
    else if ((d) <= 2048) CALL(256, 2);      \
    else if ((d) <= 8192) CALL(512, 4);      \
    else CALL(512, 8)

extern "C" {

JIB_EXPORT int jib_embed_norm(const void * table, const int * ids, const float * w, float eps, int T, int d, int n_vocab, int f32,
                              const jib_row_tail * tail, void * stream) {
    if (T <= 0) return 0;
    if (!tail_ok(tail, d)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
#define CALL(NT, MAXV)                                                                                                             \
    do {                                                                                                                           \
        if (f32) JIB_LAUNCH((embed_norm_kernel<float, NT, MAXV>), T, NT, 0, s, (const float *) table, ids, w, eps, d, n_vocab, *tail); \
        else JIB_LAUNCH((embed_norm_kernel<bf16, NT, MAXV>), T, NT, 0, s, (const bf16 *) table, ids, w, eps, d, n_vocab, *tail);       \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
    return launched();
}

JIB_EXPORT int jib_block_update(const float * x, float mult, const void * o, const void * gates, long long gate_stride, const float * b1,
                                const float * b2, const void * y, const int * dest, const float * wts, int k, int T, int d, int f32,
                                const jib_row_tail * tail, void * stream) {
    if (T <= 0) return 0;
    if (!tail_ok(tail, d) || gate_stride % 4 || (y != nullptr && (dest == nullptr || wts == nullptr || b2 == nullptr || k < 1))) return JIB_E_ARG;
    UpdateArgs a;
    a.x = x; a.o = o; a.gates = gates; a.b1 = b1; a.b2 = b2; a.y = y; a.dest = dest; a.wts = wts; a.gate_stride = gate_stride;
    a.k = k; a.d = d; a.mult = mult;
    cudaStream_t s = (cudaStream_t) stream;
    const int warm = jib::warm_for(T);
#define CALL(NT, MAXV)                                                                              \
    do {                                                                                            \
        if (f32) JIB_LAUNCH((block_update_kernel<float, NT, MAXV>), T, NT, 0, s, a, *tail, warm);   \
        else JIB_LAUNCH((block_update_kernel<bf16, NT, MAXV>), T, NT, 0, s, a, *tail, warm);        \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
    return launched();
}

JIB_EXPORT int jib_rms_rows(const float * x, const int * rows, const float * w, float eps, int n, int d, int n_src, int f32, void * out,
                            void * stream) {
    if (n <= 0) return 0;
    if (d % 4 || d > 16384 || n_src <= 0) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
#define CALL(NT, MAXV)                                                                                                       \
    do {                                                                                                                     \
        if (f32) JIB_LAUNCH((rms_rows_kernel<float, NT, MAXV>), n, NT, 0, s, x, rows, w, eps, d, n_src, (float *) out);      \
        else JIB_LAUNCH((rms_rows_kernel<bf16, NT, MAXV>), n, NT, 0, s, x, rows, w, eps, d, n_src, (bf16 *) out);            \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
    return launched();
}

}  // extern "C"
