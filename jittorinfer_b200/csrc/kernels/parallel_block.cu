// Row kernels of blocks with an fp32 residual stream.
//
// Sublayers side by side on one norm:        h = norm(x);   x <- x + m * (sigmoid(g1) * mixer(h) + sigmoid(g2) * ff(h))
// Sublayers in turn between two norms each:  x <- x + norm'(f(norm(x)))
// Sublayers side by side, a norm and a scale each:  x <- x + s1 mixer(norm1(x)) + s2 ff(norm2(x))
//
//   embed_norm     x = scale * embedding row, normed or not, then the first block's norm
//   block_update   the first form's sum -- the expert-weighted combine of the feed-forward included -- then the next block's norm
//   post_norm      the second form's sum with the norm of the sublayer's output, then the next sublayer's norm
//   scaled_update  the third form's sum, the experts' combine and a gated shared expert included, then one or two norms of the row
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

// 8 adjacent elements of a row: one 16-byte access of bf16, two of fp32.
template <typename T> struct Pack8;
template <> struct Pack8<bf16> {
    uint4 r;
    __device__ __forceinline__ void load(const bf16 * p) { r = *(const uint4 *) p; }
    __device__ __forceinline__ void zero() { r = make_uint4(0, 0, 0, 0); }
    __device__ __forceinline__ void store(bf16 * p) const { *(uint4 *) p = r; }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        const __nv_bfloat162 * h = (const __nv_bfloat162 *) &r;
#pragma unroll
        for (int i = 0; i < 4; ++i) { const float2 f = __bfloat1622float2(h[i]); v[2 * i] = f.x; v[2 * i + 1] = f.y; }
    }
    __device__ __forceinline__ void set(const float (&v)[8]) {
        __nv_bfloat162 * h = (__nv_bfloat162 *) &r;
#pragma unroll
        for (int i = 0; i < 4; ++i) h[i] = __floats2bfloat162_rn(v[2 * i], v[2 * i + 1]);
    }
};
template <> struct Pack8<float> {
    float4 a, b;
    __device__ __forceinline__ void load(const float * p) { a = ((const float4 *) p)[0]; b = ((const float4 *) p)[1]; }
    __device__ __forceinline__ void zero() { a = b = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void store(float * p) const { ((float4 *) p)[0] = a; ((float4 *) p)[1] = b; }
    __device__ __forceinline__ void get(float (&v)[8]) const {
        v[0] = a.x; v[1] = a.y; v[2] = a.z; v[3] = a.w; v[4] = b.x; v[5] = b.y; v[6] = b.z; v[7] = b.w;
    }
    __device__ __forceinline__ void set(const float (&v)[8]) { a = make_float4(v[0], v[1], v[2], v[3]); b = make_float4(v[4], v[5], v[6], v[7]); }
};
template <typename T> __device__ __forceinline__ void load8(const T * p, float (&v)[8]) {
    Pack8<T> k;
    k.load(p);
    k.get(v);
}
// bf16 activations: fast exponential and division (a few ulp of fp32); fp32 ones: the accurate forms.
template <typename T> __device__ __forceinline__ float sigmoid(float v);
template <> __device__ __forceinline__ float sigmoid<bf16>(float v) { return __fdividef(1.f, 1.f + __expf(-v)); }
template <> __device__ __forceinline__ float sigmoid<float>(float v) { return 1.f / (1.f + expf(-v)); }

constexpr int MAX_PARTS = 1024;      // equal parts of a row that a norm is taken over one by one

// 1 / rms of the part that each of a thread's vectors belongs to, from the vectors' sums of squares.  gs: NT * MAXV + MAX_PARTS floats; parts
// are whole vectors.
template <int NT, int MAXV>
__device__ __forceinline__ void part_inverses(const float (&ss)[MAXV], int d, int parts, float eps, float * gs, float (&inv)[MAXV]) {
    const int nv = d / 8, per = nv / parts;
    float * out = gs + NT * MAXV;
#pragma unroll
    for (int it = 0; it < MAXV; ++it)
        if (threadIdx.x + it * NT < nv) gs[threadIdx.x + it * NT] = ss[it];
    __syncthreads();
    for (int g = threadIdx.x >> 5; g < parts; g += NT / 32) {
        float s = 0.f;
        for (int i = threadIdx.x & 31; i < per; i += 32) s += gs[g * per + i];
        s = warp_sum(s);
        if ((threadIdx.x & 31) == 0) out[g] = rsqrtf(s / (float) (8 * per) + eps);
    }
    __syncthreads();
#pragma unroll
    for (int it = 0; it < MAXV; ++it) inv[it] = out[min((int) (threadIdx.x + it * NT) / per, parts - 1)];
}

constexpr int FAST_TAPS = 4;         // up to this many taps the stored rows are requested before the row's reductions

// x row -> residual store, norm, and (decode) the next block's input convolution.
// CONV: the tail has the convolution (decode: registers for latency); else (prompts) occupancy matters.  PARTS: the norm is taken part by
// part (gs: see part_inverses).
template <typename T, int NT, int MAXV, bool CONV, bool PARTS = false>
__device__ __forceinline__ void finish_row(float (&v)[MAXV][8], int t, int d, const jib_row_tail & a, float * red, bool dry, float * gs = nullptr) {
    const int nv = d / 8;
    constexpr bool conv = CONV;
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
    const int n_old = a.taps - 1;
    T * const state = (T *) a.conv_state + (size_t) (slot < 0 ? 0 : slot) * n_old * d;
    Pack8<T> old[MAXV == 1 && CONV ? FAST_TAPS - 1 : 1];
    const bool early = MAXV == 1 && conv && a.taps <= FAST_TAPS;
    if (early) {
#pragma unroll
        for (int j = 0; j < (MAXV == 1 && CONV ? FAST_TAPS - 1 : 0); ++j) {
            old[j].zero();
            if (past && j < n_old && threadIdx.x < nv) old[j].load(state + (size_t) j * d + 8 * threadIdx.x);
        }
    }
    float ss = 0.f, sq[MAXV], invs[MAXV];
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (PARTS) sq[it] = 0.f;
        if (i < nv) {
            Pack8<float> k;
            k.set(v[it]);
            if (!dry && a.x_out != nullptr) k.store((float *) a.x_out + (size_t) t * d + 8 * i);
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                if (PARTS) sq[it] += v[it][e] * v[it][e];
                else ss += v[it][e] * v[it][e];
            }
            if (a.norm_w == nullptr && a.h_out != nullptr && !dry) {
                Pack8<T> hp;
                hp.set(v[it]);
                hp.store((T *) a.h_out + (size_t) t * d + 8 * i);
            }
        }
    }
    if (a.norm_w == nullptr) return;
    float inv = 0.f;
    if (PARTS) {
        part_inverses<NT, MAXV>(sq, d, a.groups, a.eps, gs, invs);
    } else {
        ss = block_sum<NT>(ss, red);
        inv = rsqrtf(ss / (float) d + a.eps);
    }
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i >= nv) continue;
        if (PARTS) inv = invs[it];
        float w[8], h[8];
        load8(a.norm_w + 8 * i, w);
#pragma unroll
        for (int e = 0; e < 8; ++e) h[e] = v[it][e] * inv * w[e];
        Pack8<T> hp;
        hp.set(h);
        if (!dry) hp.store((T *) a.h_out + (size_t) t * d + 8 * i);
        if (!conv && a.norm2_w != nullptr) {
            float h2[8];
            load8(a.norm2_w + 8 * i, w);
#pragma unroll
            for (int e = 0; e < 8; ++e) h2[e] = v[it][e] * inv * w[e];
            hp.set(h2);
            if (!dry) hp.store((T *) a.h2_out + (size_t) t * d + 8 * i);
        }
        if (conv) {
            hp.get(h);                               // the convolution reads what a later step will read back from the state
            float c[8], k[8], s[8];
            load8(a.conv_w + (size_t) n_old * d + 8 * i, k);
#pragma unroll
            for (int e = 0; e < 8; ++e) c[e] = h[e] + k[e] * h[e];
            T * st = state + 8 * i;
            if (early) {
#pragma unroll
                for (int j = 0; j < (MAXV == 1 && CONV ? FAST_TAPS - 1 : 0); ++j) {
                    if (j >= n_old) continue;
                    if (past) {
                        load8(a.conv_w + (size_t) j * d + 8 * i, k);
                        old[j].get(s);
#pragma unroll
                        for (int e = 0; e < 8; ++e) c[e] += k[e] * s[e];
                    }
                    if (slot >= 0 && !dry && j > 0) old[j].store(st + (size_t) (j - 1) * d);
                }
            } else {
                for (int j = 0; j < n_old; ++j) {
                    Pack8<T> o;
                    o.zero();
                    if (past) {
                        o.load(st + (size_t) j * d);
                        load8(a.conv_w + (size_t) j * d + 8 * i, k);
                        o.get(s);
#pragma unroll
                        for (int e = 0; e < 8; ++e) c[e] += k[e] * s[e];
                    }
                    if (slot >= 0 && !dry && j > 0) o.store(st + (size_t) (j - 1) * d);
                }
            }
            if (slot >= 0 && !dry && n_old > 0) hp.store(st + (size_t) (n_old - 1) * d);
            Pack8<T> cp;
            cp.set(c);
            if (!dry) cp.store((T *) a.hc_out + (size_t) t * d + 8 * i);
        }
    }
}

template <typename T, int NT, int MAXV, bool CONV, bool PARTS>
__global__ void __launch_bounds__(NT) embed_norm_kernel(const T * __restrict__ table, const int * __restrict__ ids, const float * __restrict__ w,
                                                        float eps, float scale, int d, int n_vocab, const jib_row_tail tail) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    __shared__ float gs[PARTS ? NT * MAXV + MAX_PARTS : 1];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int t = blockIdx.x;
    int id = ids[t];
    if (id < 0 || id >= n_vocab) {
        if (threadIdx.x == 0) jib_report(tail.status, JIB_ERR_BOUNDS, 40, id);
        id = id < 0 ? 0 : n_vocab - 1;
    }
    const int nv = d / 8;
    float v[MAXV][8];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            load8(table + (size_t) id * d + 8 * i, v[it]);
#pragma unroll
            for (int e = 0; e < 8; ++e) {
                v[it][e] *= scale;
                ss += v[it][e] * v[it][e];
            }
        }
    }
    if (w != nullptr) {
        ss = block_sum<NT>(ss, red);
        const float inv = rsqrtf(ss / (float) d + eps);
#pragma unroll
        for (int it = 0; it < MAXV; ++it) {
            const int i = threadIdx.x + it * NT;
            if (i < nv) {
                float k[8];
                load8(w + 8 * i, k);
#pragma unroll
                for (int e = 0; e < 8; ++e) v[it][e] *= inv * k[e];
            }
        }
    }
    finish_row<T, NT, MAXV, CONV, PARTS>(v, t, d, tail, red, false, gs);
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

constexpr int MAX_TOP = 32;

// f = sum_j wts[j] * y[rows[j]] over 8 adjacent columns
template <typename T>
__device__ __forceinline__ void expert_sum(const T * y, const int * rows, const float * wts, int k, int d, float (&f)[8]) {
#pragma unroll
    for (int e = 0; e < 8; ++e) f[e] = 0.f;
    int j = 0;
    for (; j + 4 <= k; j += 4) {
        Pack8<T> p[4];
#pragma unroll
        for (int u = 0; u < 4; ++u) p[u].load(y + (size_t) rows[j + u] * d);
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            float q[8];
            p[u].get(q);
#pragma unroll
            for (int e = 0; e < 8; ++e) f[e] += wts[j + u] * q[e];
        }
    }
    for (; j < k; ++j) {
        float q[8];
        load8(y + (size_t) rows[j] * d, q);
#pragma unroll
        for (int e = 0; e < 8; ++e) f[e] += wts[j] * q[e];
    }
}
// a token's expert rows and weights into shared memory; all threads of the CTA
__device__ __forceinline__ void stage_pairs(const int * dest, const float * w, int k, int t, bool dry, int * rows, float * wts) {
    if (threadIdx.x < k) {
        const int r = dry ? 0 : dest[(size_t) t * k + threadIdx.x];
        rows[threadIdx.x] = r < 0 ? 0 : r;
        wts[threadIdx.x] = r < 0 ? 0.f : w == nullptr ? 1.f : w[(size_t) t * k + threadIdx.x];
    }
    __syncthreads();
}

template <typename T, int NT, int MAXV, bool CONV>
__device__ __noinline__ void block_update_row(const UpdateArgs & a, const jib_row_tail & tail, float * red, int * rows, float * wts, bool dry) {
    const int t = blockIdx.x, d = a.d, nv = d / 8;
    if (a.y != nullptr) stage_pairs(a.dest, a.wts, a.k, t, dry, rows, wts);
    float v[MAXV][8];
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i >= nv) continue;
        Pack8<float> xp, b1p, b2p;
        Pack8<T> op, g1p, g2p;
        xp.load(a.x + (size_t) t * d + 8 * i);       // everything the row needs is requested before any of it is used
        op.load((const T *) a.o + (size_t) t * d + 8 * i);
        g1p.load((const T *) a.gates + (size_t) t * a.gate_stride + 8 * i);
        b1p.load(a.b1 + 8 * i);
        float f[8], sum[8];
        if (a.y != nullptr) {
            g2p.load((const T *) a.gates + (size_t) t * a.gate_stride + d + 8 * i);
            b2p.load(a.b2 + 8 * i);
            expert_sum<T>((const T *) a.y + 8 * i, rows, wts, a.k, d, f);
        }
        float o[8], g[8], b[8], x[8];
        op.get(o); g1p.get(g); b1p.get(b); xp.get(x);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum[e] = sigmoid<T>(g[e] + b[e]) * o[e];
        if (a.y != nullptr) {
            g2p.get(g); b2p.get(b);
#pragma unroll
            for (int e = 0; e < 8; ++e) sum[e] += sigmoid<T>(g[e] + b[e]) * f[e];
        }
#pragma unroll
        for (int e = 0; e < 8; ++e) v[it][e] = x[e] + a.mult * sum[e];
    }
    finish_row<T, NT, MAXV, CONV>(v, t, d, tail, red, dry);
}

template <typename T, int NT, int MAXV, bool CONV>
__global__ void __launch_bounds__(NT, CONV || MAXV > 1 || sizeof(T) > 2 ? 1 : (1024 / NT > 1 ? 1024 / NT : 1)) block_update_kernel(const __grid_constant__ UpdateArgs a, const __grid_constant__ jib_row_tail tail, int warm) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    __shared__ int rows[MAX_TOP];
    __shared__ float wts[MAX_TOP];
    if (warm) {
        block_update_row<T, NT, MAXV, CONV>(a, tail, red, rows, wts, true);
        __syncthreads();
    }
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    block_update_row<T, NT, MAXV, CONV>(a, tail, red, rows, wts, false);
}

// x_out = x + y / rms(y) * w, then the tail's norm of it
template <typename T, int NT, int MAXV>
__device__ __noinline__ void post_norm_row(const float * x, const T * y, const float * w, float eps, int d, const jib_row_tail & tail, float * red,
                                           bool dry) {
    const int t = blockIdx.x, nv = d / 8;
    float v[MAXV][8];
    Pack8<float> xp[MAXV], wp[MAXV];
    float ss = 0.f;
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i >= nv) continue;
        Pack8<T> yp;
        yp.load(y + (size_t) t * d + 8 * i);             // everything the row needs is requested before any of it is used
        xp[it].load(x + (size_t) t * d + 8 * i);
        wp[it].load(w + 8 * i);
        yp.get(v[it]);
#pragma unroll
        for (int e = 0; e < 8; ++e) ss += v[it][e] * v[it][e];
    }
    ss = block_sum<NT>(ss, red);
    const float inv = rsqrtf(ss / (float) d + eps);
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        if (threadIdx.x + it * NT >= nv) continue;
        float k[8], r[8];
        xp[it].get(r);
        wp[it].get(k);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[it][e] = r[e] + v[it][e] * inv * k[e];
    }
    finish_row<T, NT, MAXV, false>(v, t, d, tail, red, dry);
}

template <typename T, int NT, int MAXV>
__global__ void __launch_bounds__(NT) post_norm_kernel(const float * x, const T * __restrict__ y, const float * __restrict__ w, float eps, int d,
                                                       const __grid_constant__ jib_row_tail tail, int warm) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    if (warm) {
        post_norm_row<T, NT, MAXV>(x, y, w, eps, d, tail, red, true);
        __syncthreads();
    }
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    post_norm_row<T, NT, MAXV>(x, y, w, eps, d, tail, red, false);
}

struct ScaledArgs {
    const float * x;
    const void * o, * y, * f;
    const float * s1, * s2;
    const int * dest;
    const float * wts, * f_gate;
    long long ld_gate;
    int k, d;
};

// a scale per element, or one
__device__ __forceinline__ void load_scale(Pack8<float> & p, const float * s, int c) {
    if (s != nullptr) p.load(s + c);
    else p.a = p.b = make_float4(1.f, 1.f, 1.f, 1.f);
}

template <typename T, int NT, int MAXV, bool PARTS>
__device__ __noinline__ void scaled_update_row(const ScaledArgs & a, const jib_row_tail & tail, float * red, int * rows, float * wts, float * gs,
                                               bool dry) {
    const int t = blockIdx.x, d = a.d, nv = d / 8;
    if (a.y != nullptr) stage_pairs(a.dest, a.wts, a.k, t, dry, rows, wts);
    const float g = a.f_gate != nullptr ? sigmoid<T>(a.f_gate[(size_t) t * a.ld_gate]) : 1.f;
    float v[MAXV][8];
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i >= nv) continue;
        Pack8<float> xp, s1p, s2p;
        Pack8<T> op, fp;
        xp.load(a.x + (size_t) t * d + 8 * i);       // everything the row needs is requested before any of it is used
        op.zero(); fp.zero(); s1p.zero(); s2p.zero();
        if (a.o != nullptr) {
            op.load((const T *) a.o + (size_t) t * d + 8 * i);
            load_scale(s1p, a.s1, 8 * i);
        }
        if (a.y != nullptr || a.f != nullptr) load_scale(s2p, a.s2, 8 * i);
        if (a.f != nullptr) fp.load((const T *) a.f + (size_t) t * d + 8 * i);
        float sum[8], p[8], q[8];
        if (a.y != nullptr) {
            expert_sum<T>((const T *) a.y + 8 * i, rows, wts, a.k, d, sum);
        } else {
#pragma unroll
            for (int e = 0; e < 8; ++e) sum[e] = 0.f;
        }
        fp.get(p); s2p.get(q);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum[e] = (sum[e] + g * p[e]) * q[e];
        op.get(p); s1p.get(q);
#pragma unroll
        for (int e = 0; e < 8; ++e) sum[e] += p[e] * q[e];
        xp.get(p);
#pragma unroll
        for (int e = 0; e < 8; ++e) v[it][e] = p[e] + sum[e];
    }
    finish_row<T, NT, MAXV, false, PARTS>(v, t, d, tail, red, dry, gs);
}

template <typename T, int NT, int MAXV, bool PARTS>
__global__ void __launch_bounds__(NT) scaled_update_kernel(const __grid_constant__ ScaledArgs a, const __grid_constant__ jib_row_tail tail, int warm) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    __shared__ int rows[MAX_TOP];
    __shared__ float wts[MAX_TOP];
    __shared__ float gs[PARTS ? NT * MAXV + MAX_PARTS : 1];
    if (warm) {
        scaled_update_row<T, NT, MAXV, PARTS>(a, tail, red, rows, wts, gs, true);
        __syncthreads();
    }
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    scaled_update_row<T, NT, MAXV, PARTS>(a, tail, red, rows, wts, gs, false);
}

// The row kernels for widths that 8-element vectors do not divide: element by element, the row re-read from memory.
//   ids:  v = scale * src[ids[t]], normed by w if given         (src: T table of n_src rows)
//   y:    v = x[t] + y / rms(y) * w
//   o..:  v = x[t] + the scaled sublayers of jib_scaled_update
//   else: v = x[rows[t]] (rows null: x[t])                      (x has n_src rows)
struct AnyRow {
    const void * src;
    const int * ids;
    const float * x;
    const void * y;
    const int * rows;
    const float * w;
    float eps, scale;
    int d, n_src;
    ScaledArgs u;
};
template <typename T> __device__ __forceinline__ float as_f(const void * p, size_t i);
template <> __device__ __forceinline__ float as_f<bf16>(const void * p, size_t i) { return __bfloat162float(((const bf16 *) p)[i]); }
template <> __device__ __forceinline__ float as_f<float>(const void * p, size_t i) { return ((const float *) p)[i]; }
__device__ __forceinline__ void put_f(bf16 * p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void put_f(float * p, float v) { *p = v; }

template <typename T>
__global__ void __launch_bounds__(256) any_row_kernel(const AnyRow a, const jib_row_tail tail) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    __shared__ int pair_rows[MAX_TOP];
    __shared__ float pair_wts[MAX_TOP];
    __shared__ float part_inv[MAX_PARTS];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int t = blockIdx.x, d = a.d;
    const ScaledArgs & u = a.u;
    if (u.y != nullptr) stage_pairs(u.dest, u.wts, u.k, t, false, pair_rows, pair_wts);
    const float gate = u.f_gate != nullptr ? sigmoid<T>(u.f_gate[(size_t) t * u.ld_gate]) : 1.f;
    size_t row = t;
    if (a.ids != nullptr || a.rows != nullptr) {
        int r = a.ids != nullptr ? a.ids[t] : a.rows[t];
        if (r < 0 || r >= a.n_src) {
            if (threadIdx.x == 0 && a.ids != nullptr) jib_report(tail.status, JIB_ERR_BOUNDS, 40, r);
            r = r < 0 ? 0 : a.n_src - 1;
        }
        row = r;
    }
    const void * normed = a.ids != nullptr ? a.src : a.y;        // the operand that w belongs to
    float inv = 1.f;
    if (normed != nullptr && a.w != nullptr) {
        float ss = 0.f;
        for (int i = threadIdx.x; i < d; i += 256) {
            const float v = a.scale * as_f<T>(normed, row * d + i);
            ss += v * v;
        }
        inv = rsqrtf(block_sum<256>(ss, red) / (float) d + a.eps);
    }
    auto value = [&](int i) {
        float v = 0.f;
        if (normed != nullptr) {
            v = a.scale * as_f<T>(normed, row * d + i);
            if (a.w != nullptr) v *= inv * a.w[i];
        }
        if (u.y != nullptr || u.f != nullptr) {
            float f = u.f != nullptr ? gate * as_f<T>(u.f, row * d + i) : 0.f;
            if (u.y != nullptr)
                for (int j = 0; j < u.k; ++j) f += pair_wts[j] * as_f<T>(u.y, (size_t) pair_rows[j] * d + i);
            v += (u.s2 != nullptr ? u.s2[i] : 1.f) * f;
        }
        if (u.o != nullptr) v += (u.s1 != nullptr ? u.s1[i] : 1.f) * as_f<T>(u.o, row * d + i);
        return a.x != nullptr ? v + a.x[row * d + i] : v;
    };
    float * xo = (float *) tail.x_out;
    float ss = 0.f;
    const int parts = tail.norm_w != nullptr && tail.groups > 1 ? tail.groups : 1, part = d / parts;
    for (int i = threadIdx.x; i < d; i += 256) {
        if (parts > 1) break;
        const float v = value(i);
        ss += v * v;
        if (tail.norm_w == nullptr && tail.h_out != nullptr) put_f((T *) tail.h_out + (size_t) t * d + i, v);
        if (tail.norm_w == nullptr && xo != nullptr) xo[(size_t) t * d + i] = v;
    }
    if (tail.norm_w == nullptr) return;
    if (parts > 1) {
        for (int g = threadIdx.x >> 5; g < parts; g += 8) {
            float s = 0.f;
            for (int i = threadIdx.x & 31; i < part; i += 32) {
                const float v = value(g * part + i);
                s += v * v;
            }
            s = warp_sum(s);
            if ((threadIdx.x & 31) == 0) part_inv[g] = rsqrtf(s / (float) part + tail.eps);
        }
        __syncthreads();
    } else {
        ss = block_sum<256>(ss, red);
    }
    const float all_inv = rsqrtf(ss / (float) d + tail.eps);
    for (int i = threadIdx.x; i < d; i += 256) {
        const float v = value(i), ni = parts > 1 ? part_inv[i / part] : all_inv;
        put_f((T *) tail.h_out + (size_t) t * d + i, v * ni * tail.norm_w[i]);
        if (tail.norm2_w != nullptr) put_f((T *) tail.h2_out + (size_t) t * d + i, v * ni * tail.norm2_w[i]);
        if (xo != nullptr) xo[(size_t) t * d + i] = v;            // last: x_out may be x
    }
}

// out[i] = x[rows[i]] / rms * w
template <typename T, int NT, int MAXV, bool PARTS>
__global__ void __launch_bounds__(NT) rms_rows_kernel(const float * __restrict__ x, const int * __restrict__ rows, const float * __restrict__ w,
                                                      float eps, int d, int n_src, int parts, T * __restrict__ out) {
    PDL_TRIGGER_TOP();
    __shared__ float red[32];
    __shared__ float gs[PARTS ? NT * MAXV + MAX_PARTS : 1];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int r = rows != nullptr ? rows[blockIdx.x] : (int) blockIdx.x;
    r = r < 0 ? 0 : (r >= n_src ? n_src - 1 : r);
    const int nv = d / 8;
    float v[MAXV][8];
    float ss = 0.f, sq[MAXV], invs[MAXV];
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        sq[it] = 0.f;
        if (i < nv) {
            load8(x + (size_t) r * d + 8 * i, v[it]);
#pragma unroll
            for (int e = 0; e < 8; ++e) sq[it] += v[it][e] * v[it][e];
        }
        ss += sq[it];
    }
    float inv = 0.f;
    if (PARTS) {
        part_inverses<NT, MAXV>(sq, d, parts, eps, gs, invs);
    } else {
        ss = block_sum<NT>(ss, red);
        inv = rsqrtf(ss / (float) d + eps);
    }
#pragma unroll
    for (int it = 0; it < MAXV; ++it) {
        const int i = threadIdx.x + it * NT;
        if (i < nv) {
            if (PARTS) inv = invs[it];
            float k[8];
            load8(w + 8 * i, k);
#pragma unroll
            for (int e = 0; e < 8; ++e) v[it][e] *= inv * k[e];
            Pack8<T> o;
            o.set(v[it]);
            o.store(out + (size_t) blockIdx.x * d + 8 * i);
        }
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

inline bool tail_ok(const jib_row_tail * t, int d) {
    if (t == nullptr || t->x_out == nullptr || d > 16384) return false;
    if (t->norm2_w != nullptr && (t->norm_w == nullptr || t->h2_out == nullptr || t->conv_w != nullptr)) return false;
    if (t->groups > 1 && (t->groups > MAX_PARTS || d % t->groups || t->conv_w != nullptr)) return false;
    if (d % 8) return t->conv_w == nullptr && (t->norm_w == nullptr || t->h_out != nullptr);      // the element-wise kernel
    if (t->norm_w != nullptr && t->h_out == nullptr) return false;
    if (t->conv_w != nullptr)
        return t->norm_w != nullptr && t->hc_out != nullptr && t->taps >= 1 && (t->taps == 1 || t->conv_state != nullptr) &&
               t->seq_slots != nullptr && t->positions != nullptr && t->n_state >= 0;
    return true;
}
// rows (or parts of rows) that 8-element vectors do not divide take the element-wise kernel
inline bool by_element(int d, int parts) { return d % 8 || (parts > 1 && d / parts % 8); }

}  // namespace

// (threads, 8-element vectors per thread) by row width
#define JIB_ROW_DISPATCH(d, CALL)            \
    if ((d) <= 1024) CALL(128, 1);           \
    else if ((d) <= 2048) CALL(256, 1);      \
    else if ((d) <= 4096) CALL(512, 1);      \
    else if ((d) <= 5120) CALL(640, 1);      \
    else if ((d) <= 8192) CALL(512, 2);      \
    else CALL(512, 4)

extern "C" {

static int launch_any(const AnyRow & a, const jib_row_tail & tail, int n, int f32, cudaStream_t s) {
    if (f32) JIB_LAUNCH((any_row_kernel<float>), n, 256, 0, s, a, tail);
    else JIB_LAUNCH((any_row_kernel<bf16>), n, 256, 0, s, a, tail);
    return launched();
}

JIB_EXPORT int jib_embed_norm(const void * table, const int * ids, const float * w, float eps, float scale, int T, int d, int n_vocab, int f32,
                              const jib_row_tail * tail, void * stream) {
    if (T <= 0) return 0;
    if (!tail_ok(tail, d)) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    if (by_element(d, tail->groups)) {
        AnyRow a = {};
        a.src = table; a.ids = ids; a.w = w; a.eps = eps; a.scale = scale; a.d = d; a.n_src = n_vocab;
        return launch_any(a, *tail, T, f32, s);
    }
#define EMBED(TT, NT, MAXV, CONV, PARTS) \
    JIB_LAUNCH((embed_norm_kernel<TT, NT, MAXV, CONV, PARTS>), T, NT, 0, s, (const TT *) table, ids, w, eps, scale, d, n_vocab, *tail)
#define CALL(NT, MAXV)                                                    \
    do {                                                                  \
        if (tail->conv_w != nullptr) {                                    \
            if (f32) EMBED(float, NT, MAXV, true, false);                 \
            else EMBED(bf16, NT, MAXV, true, false);                      \
        } else if (tail->groups > 1) {                                    \
            if (f32) EMBED(float, NT, MAXV, false, true);                 \
            else EMBED(bf16, NT, MAXV, false, true);                      \
        } else {                                                          \
            if (f32) EMBED(float, NT, MAXV, false, false);                \
            else EMBED(bf16, NT, MAXV, false, false);                     \
        }                                                                 \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
#undef EMBED
    return launched();
}

JIB_EXPORT int jib_block_update(const float * x, float mult, const void * o, const void * gates, long long gate_stride, const float * b1,
                                const float * b2, const void * y, const int * dest, const float * wts, int k, int T, int d, int f32,
                                const jib_row_tail * tail, void * stream) {
    if (T <= 0) return 0;
    if (!tail_ok(tail, d) || tail->groups > 1 || d % 8 || gate_stride % 8 || (y != nullptr && (dest == nullptr || wts == nullptr || b2 == nullptr || k < 1 || k > MAX_TOP))) return JIB_E_ARG;
    UpdateArgs a;
    a.x = x; a.o = o; a.gates = gates; a.b1 = b1; a.b2 = b2; a.y = y; a.dest = dest; a.wts = wts; a.gate_stride = gate_stride;
    a.k = k; a.d = d; a.mult = mult;
    cudaStream_t s = (cudaStream_t) stream;
    const int warm = jib::warm_for(T);
#define UPDATE(TT, NT, MAXV, CONV) JIB_LAUNCH((block_update_kernel<TT, NT, MAXV, CONV>), T, NT, 0, s, a, *tail, warm)
#define CALL(NT, MAXV)                                                    \
    do {                                                                  \
        if (tail->conv_w != nullptr) {                                    \
            if (f32) UPDATE(float, NT, MAXV, true);                       \
            else UPDATE(bf16, NT, MAXV, true);                            \
        } else {                                                          \
            if (f32) UPDATE(float, NT, MAXV, false);                      \
            else UPDATE(bf16, NT, MAXV, false);                           \
        }                                                                 \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
#undef UPDATE
    return launched();
}

JIB_EXPORT int jib_post_norm(const float * x, const void * y, const float * w, float eps, int T, int d, int f32, const jib_row_tail * tail,
                             void * stream) {
    if (T <= 0) return 0;
    if (!tail_ok(tail, d) || tail->groups > 1 || tail->conv_w != nullptr || w == nullptr) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    if (d % 8) {
        AnyRow a = {};
        a.x = x; a.y = y; a.w = w; a.eps = eps; a.scale = 1.f; a.d = d; a.n_src = T;
        return launch_any(a, *tail, T, f32, s);
    }
    const int warm = jib::warm_for(T);
#define CALL(NT, MAXV)                                                                                                          \
    do {                                                                                                                        \
        if (f32) JIB_LAUNCH((post_norm_kernel<float, NT, MAXV>), T, NT, 0, s, x, (const float *) y, w, eps, d, *tail, warm);    \
        else JIB_LAUNCH((post_norm_kernel<bf16, NT, MAXV>), T, NT, 0, s, x, (const bf16 *) y, w, eps, d, *tail, warm);          \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
    return launched();
}

JIB_EXPORT int jib_scaled_update(const float * x, const void * o, const float * s1, const void * y, const int * dest, const float * wts, int k,
                                 const void * f, const float * f_gate, long long ld_gate, const float * s2, int T, int d, int f32,
                                 const jib_row_tail * tail, void * stream) {
    if (T <= 0) return 0;
    jib_row_tail chk = *tail;
    if (chk.x_out == nullptr) chk.x_out = (void *) x;
    if (!tail_ok(&chk, d) || tail->conv_w != nullptr || (y != nullptr && (dest == nullptr || k < 1 || k > MAX_TOP)))
        return JIB_E_ARG;
    ScaledArgs a;
    a.x = x; a.o = o; a.y = y; a.f = f; a.s1 = s1; a.s2 = s2; a.dest = dest; a.wts = wts; a.f_gate = f_gate; a.ld_gate = ld_gate;
    a.k = k; a.d = d;
    cudaStream_t s = (cudaStream_t) stream;
    if (by_element(d, tail->groups)) {
        AnyRow r = {};
        r.x = x; r.d = d; r.n_src = T; r.scale = 1.f; r.u = a;
        return launch_any(r, *tail, T, f32, s);
    }
    const int warm = jib::warm_for(T);
#define UPDATE(TT, NT, MAXV, PARTS) JIB_LAUNCH((scaled_update_kernel<TT, NT, MAXV, PARTS>), T, NT, 0, s, a, *tail, warm)
#define CALL(NT, MAXV)                                                    \
    do {                                                                  \
        if (tail->norm_w != nullptr && tail->groups > 1) {                \
            if (f32) UPDATE(float, NT, MAXV, true);                       \
            else UPDATE(bf16, NT, MAXV, true);                            \
        } else {                                                          \
            if (f32) UPDATE(float, NT, MAXV, false);                      \
            else UPDATE(bf16, NT, MAXV, false);                           \
        }                                                                 \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
#undef UPDATE
    return launched();
}

JIB_EXPORT int jib_rms_rows(const float * x, const int * rows, const float * w, float eps, int n, int d, int n_src, int groups, int f32, void * out,
                            void * stream) {
    if (n <= 0) return 0;
    if (d > 16384 || n_src <= 0 || groups < 1 || groups > MAX_PARTS || d % groups) return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    if (by_element(d, groups)) {
        AnyRow a = {};
        jib_row_tail t = {};
        a.x = x; a.rows = rows; a.d = d; a.n_src = n_src; a.scale = 1.f;
        t.norm_w = w; t.eps = eps; t.h_out = out; t.groups = groups;
        return launch_any(a, t, n, f32, s);
    }
#define ROWS(TT, NT, MAXV, PARTS) JIB_LAUNCH((rms_rows_kernel<TT, NT, MAXV, PARTS>), n, NT, 0, s, x, rows, w, eps, d, n_src, groups, (TT *) out)
#define CALL(NT, MAXV)                                                    \
    do {                                                                  \
        if (groups > 1) {                                                 \
            if (f32) ROWS(float, NT, MAXV, true);                         \
            else ROWS(bf16, NT, MAXV, true);                              \
        } else {                                                          \
            if (f32) ROWS(float, NT, MAXV, false);                        \
            else ROWS(bf16, NT, MAXV, false);                             \
        }                                                                 \
    } while (0)
    JIB_ROW_DISPATCH(d, CALL);
#undef CALL
#undef ROWS
    return launched();
}

}  // extern "C"
