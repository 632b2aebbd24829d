// Selective scan: every channel c carries N states with a decay of their own,
//
//   S[c][n] <- exp(dt_c a[c][n]) S[c][n] + dt_c x_c B_n;   y_c = (sum_n S[c][n] C_n + skip_c x_c) * silu(z_c) * out_scale
//
// with dt = softplus(dt_c + bias_c) and B, C shared by the channels.  L lanes of a warp share a channel, NS states each.
//
//   scan_step      one token per sequence: the state is read and written once, several sequences per thread in flight
//   scan_portions  ranges of any length: a CTA owns 128 / L channels of one sequence, keeps their states in registers and walks the
//                  tokens in tiles of TT, the next tile's inputs on their way while one is worked on
//
// The exponentials do not depend on the state, so a token costs its lane one multiply-add of latency.  Tokens go in groups of 8: while
// a group's recurrence runs the next one's decays and inputs are computed, and the lanes' partial sums meet in one butterfly that
// leaves each lane with the sums of some of the tokens.  A bf16 tile is one straight line of code.  Shared memory's bandwidth is the
// tightest resource (a load moves a warp's full width even where lanes share an address), so B and C stay bf16 there.
//
// A sequence's state lives in row seq_slots[b] of [n_state][ch][N]; a range that starts at position 0 starts from zeros whatever the
// row holds.  Sequence b owns token rows q_start[b] .. q_start[b + 1].  Activations bf16 or fp32, the rest fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "pdl.cuh"
#include "sm100.cuh"

namespace {

typedef __nv_bfloat16 bf16;

constexpr int NT = 128;                                      // threads of a CTA

__device__ __forceinline__ float to_f(bf16 v) { return __bfloat162float(v); }
__device__ __forceinline__ float to_f(float v) { return v; }
__device__ __forceinline__ void put(bf16 * p, float v) { *p = __float2bfloat16(v); }
__device__ __forceinline__ void put(float * p, float v) { *p = v; }
// bf16 activations: fast exponential and division for the gate, a base-2 exponential for the decays; fp32 ones: the accurate forms.
template <typename T> __device__ __forceinline__ float silu(float v);
template <> __device__ __forceinline__ float silu<bf16>(float v) { return v * __fdividef(1.f, 1.f + __expf(-v)); }
template <> __device__ __forceinline__ float silu<float>(float v) { return v / (1.f + expf(-v)); }
template <typename T> __device__ __forceinline__ float rate(float neg_a);            // what advance() takes, times dt
template <> __device__ __forceinline__ float rate<bf16>(float neg_a) { return neg_a * 1.4426950408889634f; }
template <> __device__ __forceinline__ float rate<float>(float neg_a) { return neg_a; }
// exp(v) s + u, v <= 0.  fp32: a decay close to 1 as s + s (exp(v) - 1), or its rounding to 24 bits would bias every step alike
template <typename T> __device__ __forceinline__ float advance(float v, float s, float u);
template <> __device__ __forceinline__ float advance<bf16>(float v, float s, float u) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r * s + u;
}
template <> __device__ __forceinline__ float advance<float>(float v, float s, float u) {
    return (v > -0.5f ? fmaf(s, expm1f(v), s) : s * expf(v)) + u;
}
// log(1 + e^v) = max(v, 0) + log1p(e^-|v|).  bf16: log1p(e) = 2 atanh(r), r = e / (2 + e) <= 1/3, by atanh's series to r^13 (relative
// error below 1e-7).
template <typename T> __device__ __forceinline__ float softplus(float v);
template <> __device__ __forceinline__ float softplus<float>(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }
template <> __device__ __forceinline__ float softplus<bf16>(float v) {
    const float e = __expf(-fabsf(v)), r = __fdividef(e, 2.f + e), q = r * r;
    float p = q * (2.f / 13.f) + 2.f / 11.f;
    p = p * q + 2.f / 9.f;
    p = p * q + 2.f / 7.f;
    p = p * q + 2.f / 5.f;
    p = p * q + 2.f / 3.f;
    p = p * q + 2.f;
    return fmaxf(v, 0.f) + p * r;
}
// two fp32 operations per instruction
struct F2 {
    unsigned long long v;
};
__device__ __forceinline__ F2 pack(float a, float b) {
    F2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r.v) : "f"(a), "f"(b));
    return r;
}
__device__ __forceinline__ float2 unpack(F2 a) {
    float2 r;
    asm("mov.b64 {%0, %1}, %2;" : "=f"(r.x), "=f"(r.y) : "l"(a.v));
    return r;
}
__device__ __forceinline__ F2 fma2(F2 a, F2 b, F2 c) {
    F2 r;
    asm("fma.rn.f32x2 %0, %1, %2, %3;" : "=l"(r.v) : "l"(a.v), "l"(b.v), "l"(c.v));
    return r;
}
__device__ __forceinline__ F2 mul2(F2 a, F2 b) {
    F2 r;
    asm("mul.rn.f32x2 %0, %1, %2;" : "=l"(r.v) : "l"(a.v), "l"(b.v));
    return r;
}
// the decays of two states, and their next values; fp32 decays are kept as the exponent (see advance)
template <typename T> __device__ __forceinline__ F2 decay2(F2 v);
template <> __device__ __forceinline__ F2 decay2<bf16>(F2 v) {
    float2 e = unpack(v);
    asm("ex2.approx.ftz.f32 %0, %0;" : "+f"(e.x));
    asm("ex2.approx.ftz.f32 %0, %0;" : "+f"(e.y));
    return pack(e.x, e.y);
}
template <> __device__ __forceinline__ F2 decay2<float>(F2 v) { return v; }
template <typename T> __device__ __forceinline__ F2 next2(F2 e, F2 s, F2 u);
template <> __device__ __forceinline__ F2 next2<bf16>(F2 e, F2 s, F2 u) { return fma2(e, s, u); }
template <> __device__ __forceinline__ F2 next2<float>(F2 e, F2 s, F2 u) {
    const float2 v = unpack(e), x = unpack(s), y = unpack(u);
    return pack(advance<float>(v.x, x.x, y.x), advance<float>(v.y, x.y, y.y));
}

// 4 adjacent elements, kept as stored until they are needed (many loads in flight)
template <typename T> struct Quad;
template <> struct Quad<float> {
    float4 r;
    __device__ __forceinline__ void zero() { r = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void load(const float * p) { r = *(const float4 *) p; }
    // not moved towards the use
    __device__ __forceinline__ void request(const float * p) {
        asm volatile("ld.global.v4.f32 {%0, %1, %2, %3}, [%4];" : "=f"(r.x), "=f"(r.y), "=f"(r.z), "=f"(r.w) : "l"(p));
    }
    __device__ __forceinline__ float4 get() const { return r; }
    __device__ __forceinline__ static void store(float * p, float4 v) { *(float4 *) p = v; }
};
template <> struct Quad<bf16> {
    uint2 r;
    __device__ __forceinline__ void zero() { r = make_uint2(0, 0); }
    __device__ __forceinline__ void load(const bf16 * p) { r = *(const uint2 *) p; }
    __device__ __forceinline__ void request(const bf16 * p) { asm volatile("ld.global.v2.u32 {%0, %1}, [%2];" : "=r"(r.x), "=r"(r.y) : "l"(p)); }
    __device__ __forceinline__ float4 get() const {
        const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *) &r.x), y = __bfloat1622float2(*(const __nv_bfloat162 *) &r.y);
        return make_float4(x.x, x.y, y.x, y.y);
    }
    __device__ __forceinline__ static void store(bf16 * p, float4 v) {
        uint2 o;
        *(__nv_bfloat162 *) &o.x = __floats2bfloat162_rn(v.x, v.y);
        *(__nv_bfloat162 *) &o.y = __floats2bfloat162_rn(v.z, v.w);
        *(uint2 *) p = o;
    }
};
// NS adjacent floats, NS 2 or a multiple of 4
template <int NS> __device__ __forceinline__ void load_n(const float * p, float (&v)[NS]) {
    if constexpr (NS == 2) {
        const float2 x = *(const float2 *) p;
        v[0] = x.x; v[1] = x.y;
    } else {
#pragma unroll
        for (int i = 0; i < NS; i += 4) {
            const float4 x = *(const float4 *) (p + i);
            v[i] = x.x; v[i + 1] = x.y; v[i + 2] = x.z; v[i + 3] = x.w;
        }
    }
}
template <int NS> __device__ __forceinline__ void store_n(float * p, const float (&v)[NS]) {
    if constexpr (NS == 2) {
        *(float2 *) p = make_float2(v[0], v[1]);
    } else {
#pragma unroll
        for (int i = 0; i < NS; i += 4) *(float4 *) (p + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
    }
}
template <int H> __device__ __forceinline__ void load_pairs(const float * p, F2 (&v)[H]) {
    if constexpr (H == 1) {
        v[0].v = *(const unsigned long long *) p;
    } else {
#pragma unroll
        for (int i = 0; i < H; i += 2) {
            const ulonglong2 x = *(const ulonglong2 *) (p + 2 * i);
            v[i].v = x.x;
            v[i + 1].v = x.y;
        }
    }
}

// B and C of a tile in shared memory, a lane's NS states of both adjacent (row: L times NS of B, NS of C), as stored: bf16 halves the traffic
template <typename T, int NS> struct Operands;
template <int NS> struct Operands<float, NS> {
    static __device__ __forceinline__ void put(float * row, int col, bool is_c, const Quad<float> & v) {
        const float x[4] = {v.r.x, v.r.y, v.r.z, v.r.w};
#pragma unroll
        for (int i = 0; i < 4; i += 2) *(float2 *) (row + (col + i) / NS * 2 * NS + (is_c ? NS : 0) + (col + i) % NS) = make_float2(x[i], x[i + 1]);
    }
    static __device__ __forceinline__ void get(const float * p, F2 (&B)[NS / 2], F2 (&C)[NS / 2]) {
        load_pairs<NS / 2>(p, B);
        load_pairs<NS / 2>(p + NS, C);
    }
};
template <int NS> struct Operands<bf16, NS> {
    static __device__ __forceinline__ void put(bf16 * row, int col, bool is_c, const Quad<bf16> & v) {
        *(uint32_t *) (row + col / NS * 2 * NS + (is_c ? NS : 0) + col % NS) = v.r.x;
        *(uint32_t *) (row + (col + 2) / NS * 2 * NS + (is_c ? NS : 0) + (col + 2) % NS) = v.r.y;
    }
    static __device__ __forceinline__ void get(const bf16 * p, F2 (&B)[NS / 2], F2 (&C)[NS / 2]) {
        uint32_t r[NS];
        if constexpr (NS == 2) {
            const uint2 x = *(const uint2 *) p;
            r[0] = x.x; r[1] = x.y;
        } else {
#pragma unroll
            for (int i = 0; i < NS; i += 4) {
                const uint4 x = *(const uint4 *) (p + 2 * i);
                r[i] = x.x; r[i + 1] = x.y; r[i + 2] = x.z; r[i + 3] = x.w;
            }
        }
#pragma unroll
        for (int i = 0; i < NS / 2; ++i) {
            B[i] = pack(__uint_as_float(r[i] << 16), __uint_as_float(r[i] & 0xffff0000u));
            C[i] = pack(__uint_as_float(r[NS / 2 + i] << 16), __uint_as_float(r[NS / 2 + i] & 0xffff0000u));
        }
    }
};

__device__ __forceinline__ int checked_slot(const jib_scan & a, int b, int site) {
    const int slot = a.seq_slots[b];
    if (slot >= a.n_state) {
        if (threadIdx.x == 0) jib_report(a.status, JIB_ERR_BOUNDS, site, slot);
        return -1;
    }
    return slot;
}

// ---- single tokens: grid (ceil(ch / (NT / L)), ceil(T / U)), row t belongs to sequence t ---------------------------------------------
template <typename T, int NS, int L, int U>
__global__ void __launch_bounds__(NT) scan_step_kernel(const __grid_constant__ jib_scan a) {
    PDL_TRIGGER_TOP();
    const int lane = threadIdx.x % L, c = blockIdx.x * (NT / L) + threadIdx.x / L, n0 = lane * NS;
    const bool mine = c < a.ch, live = mine && n0 < a.N;
    const int cc = mine ? c : a.ch - 1, nn = n0 < a.N ? n0 : 0;
    float ra[NS];
    load_n<NS>(a.neg_a + (size_t) cc * a.N + nn, ra);        // launch-invariant
    const float skip = a.skip[cc], bias = a.dt_bias[cc];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int slot[U];
    float s[U][NS], dt[U], x[U], z[U];
    Quad<T> B[U][NS / 4], C[U][NS / 4];
#pragma unroll
    for (int u = 0; u < U; ++u) {                            // everything the rows need is requested before any of it is used
        const int t = blockIdx.y * U + u, tt = min(t, a.T - 1);
        slot[u] = t < a.T ? checked_slot(a, t, 51) : -1;
#pragma unroll
        for (int i = 0; i < NS; ++i) s[u][i] = 0.f;
        if (slot[u] >= 0 && live && a.positions[tt] > 0) load_n<NS>(a.state + ((size_t) slot[u] * a.ch + cc) * a.N + nn, s[u]);
        const T * bc = (const T *) a.bc + (size_t) tt * a.ldbc + nn;
#pragma unroll
        for (int i = 0; i < NS / 4; ++i) {
            B[u][i].load(bc + 4 * i);
            C[u][i].load(bc + a.N + 4 * i);
        }
        x[u] = to_f(((const T *) a.x)[(size_t) tt * a.ldx + cc]);
        z[u] = to_f(((const T *) a.z)[(size_t) tt * a.ldz + cc]);
        dt[u] = to_f(((const T *) a.dt)[(size_t) tt * a.lddt + cc]);
    }
#pragma unroll
    for (int i = 0; i < NS; ++i) ra[i] = rate<T>(ra[i]);
#pragma unroll
    for (int u = 0; u < U; ++u) {
        const int t = blockIdx.y * U + u;
        const float d = softplus<T>(dt[u] + bias), dx = d * x[u];
        float y = 0.f;
#pragma unroll
        for (int i = 0; i < NS / 4; ++i) {
            const float4 b = B[u][i].get(), k = C[u][i].get();
            const float bv[4] = {b.x, b.y, b.z, b.w}, kv[4] = {k.x, k.y, k.z, k.w};
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                s[u][4 * i + e] = advance<T>(d * ra[4 * i + e], s[u][4 * i + e], dx * bv[e]);
                y += s[u][4 * i + e] * kv[e];
            }
        }
        if (!live) y = 0.f;
        if (live && slot[u] >= 0) store_n<NS>(a.state + ((size_t) slot[u] * a.ch + cc) * a.N + nn, s[u]);
#pragma unroll
        for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
        if (lane == 0 && mine && t < a.T) put((T *) a.y + (size_t) t * a.ldy + c, (y + skip * x[u]) * silu<T>(z[u]) * a.out_scale);
    }
}

// ---- portions: grid (ceil(ch / CH), n_seqs) ----------------------------------------------------------------------------------------
template <typename T, int NS, int L>
struct Scan {
    static constexpr int NP = NS * L, CH = NT / L;
    static constexpr int TT = NP <= 64 ? 32 : 8;             // tokens of a tile
    static constexpr int G = 8;                              // tokens of a group
    static constexpr int QX = TT * CH / 4, QB = TT * 2 * NP / 4;                     // quads of a tile: per channel input, of B | C
    static constexpr int RX = (QX + NT - 1) / NT, RB = (QB + NT - 1) / NT;
    static constexpr int SMEM = TT * CH * 8 + TT * 2 * NP * (int) sizeof(T) + TT * CH * 4;
    Quad<T> x[RX], z[RX], dt[RX], bc[RB];
    // tokens t0 .. of the sequence's n, whose first row is q0
    __device__ __forceinline__ void load(const jib_scan & a, int q0, int n, int t0, int c0) {
#pragma unroll
        for (int i = 0; i < RX; ++i) {
            const int q = threadIdx.x + i * NT, t = t0 + q / (CH / 4), c = c0 + q % (CH / 4) * 4;
            x[i].zero(); z[i].zero(); dt[i].zero();
            if (q < QX && t < n && c < a.ch) {
                const size_t r = q0 + t;
                x[i].request((const T *) a.x + r * a.ldx + c);
                z[i].request((const T *) a.z + r * a.ldz + c);
                dt[i].request((const T *) a.dt + r * a.lddt + c);
            }
        }
        const int n4 = a.N / 2;                              // quads of a row of B | C
#pragma unroll
        for (int i = 0; i < RB; ++i) {
            const int q = threadIdx.x + i * NT, k = q / n4, t = t0 + k;
            bc[i].zero();
            if (k < TT && t < n) bc[i].request((const T *) a.bc + (size_t) (q0 + t) * a.ldbc + (q - k * n4) * 4);
        }
    }
};

// The L lanes' partial sums of 8 tokens -> lane j < W holds those of tokens j * 8 / W .. in p[0 .. 8 / W), W = min(L, 8).
template <int L> __device__ __forceinline__ void meet(float (&p)[8], int lane) {
    constexpr int W = L < 8 ? L : 8;
    int n = 8;
#pragma unroll
    for (int o = W / 2; o > 0; o >>= 1) {
        n >>= 1;
        const bool up = (lane & o) != 0;
#pragma unroll
        for (int k = 0; k < 4; ++k) {
            if (k >= n) break;
            const float keep = up ? p[k + n] : p[k], send = up ? p[k] : p[k + n];
            p[k] = keep + __shfl_xor_sync(0xffffffffu, send, o);
        }
    }
#pragma unroll
    for (int o = W; o < L; o <<= 1) p[0] += __shfl_xor_sync(0xffffffffu, p[0], o);
}

template <typename T, int NS, int L>
__global__ void __launch_bounds__(NT, NS >= 8 ? 1 : 3) scan_portions_kernel(const __grid_constant__ jib_scan a) {
    using S = Scan<T, NS, L>;
    constexpr int NP = S::NP, CH = S::CH, TT = S::TT, G = S::G, W = L < 8 ? L : 8, H = NS / 2;
    extern __shared__ __align__(16) float smem[];
    float2 * sdx = (float2 *) smem;                          // [TT][CH]: step size, step size * x
    float * sy = smem + TT * CH * 2;                         // [TT][CH]
    T * sbc = (T *) (sy + TT * CH);                          // [TT][2 NP], see Operands
    PDL_TRIGGER_TOP();
    const int lane = threadIdx.x % L, cl = threadIdx.x / L, c0 = blockIdx.x * CH, c = c0 + cl, b = blockIdx.y, n0 = lane * NS;
    const bool live = c < a.ch && n0 < a.N;
    F2 ra[H], s[H];
    {
        float v[NS];
#pragma unroll
        for (int i = 0; i < NS; ++i) v[i] = 0.f;
        if (live) load_n<NS>(a.neg_a + (size_t) c * a.N + n0, v);
#pragma unroll
        for (int i = 0; i < H; ++i) ra[i] = pack(rate<T>(v[2 * i]), rate<T>(v[2 * i + 1]));
    }
    for (int i = threadIdx.x; i < TT * 2 * NP; i += NT) put(sbc + i, 0.f);           // columns past N stay zero
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int q0 = a.q_start[b], n = a.q_start[b + 1] - q0;
    if (n <= 0) return;
    S cur, nxt;
    cur.load(a, q0, n, 0, c0);
    const int slot = checked_slot(a, b, 52);
    float * st = a.state + ((size_t) (slot < 0 ? 0 : slot) * a.ch + c) * a.N + n0;
    {
        float v[NS];
#pragma unroll
        for (int i = 0; i < NS; ++i) v[i] = 0.f;
        if (live && slot >= 0 && a.positions[q0] > 0) load_n<NS>(st, v);
#pragma unroll
        for (int i = 0; i < H; ++i) s[i] = pack(v[2 * i], v[2 * i + 1]);
    }
    const int cq = threadIdx.x % (CH / 4) * 4;               // this thread's quads: the same channels of different tokens
    static_assert(NT % (CH / 4) == 0, "");
    float4 skip = make_float4(0.f, 0.f, 0.f, 0.f), bias = skip;
    if (c0 + cq < a.ch) {
        skip = *(const float4 *) (a.skip + c0 + cq);
        bias = *(const float4 *) (a.dt_bias + c0 + cq);
    }
    __syncthreads();
    for (int t0 = 0; t0 < n; t0 += TT) {
#pragma unroll
        for (int i = 0; i < S::RX; ++i) {
            const int q = threadIdx.x + i * NT, t = q / (CH / 4);
            if (q >= S::QX) continue;
            const float4 x = cur.x[i].get(), d = cur.dt[i].get();
            const float xv[4] = {x.x, x.y, x.z, x.w}, dv[4] = {d.x + bias.x, d.y + bias.y, d.z + bias.z, d.w + bias.w};
            float k[4];
#pragma unroll
            for (int e = 0; e < 4; ++e) k[e] = t0 + t < n ? softplus<T>(dv[e]) : 0.f;   // past the end: the state passes through
            float4 * o = (float4 *) (sdx + t * CH + cq);
            o[0] = make_float4(k[0], k[0] * xv[0], k[1], k[1] * xv[1]);
            o[1] = make_float4(k[2], k[2] * xv[2], k[3], k[3] * xv[3]);
        }
        const int n4 = a.N / 2;
#pragma unroll
        for (int i = 0; i < S::RB; ++i) {
            const int q = threadIdx.x + i * NT, t = q / n4, col = (q - t * n4) * 4;
            if (t < TT) Operands<T, NS>::put(sbc + t * 2 * NP, col < a.N ? col : col - a.N, col >= a.N, cur.bc[i]);
        }
        __syncthreads();
        if (t0 + TT < n) nxt.load(a, q0, n, t0 + TT, c0);
        const int m = min(TT, n - t0);
        // decays, inputs and read-out weights of token t
        auto prepare = [&](int t, F2 (&e)[H], F2 (&u)[H], F2 (&C)[H]) {
            const float2 d = sdx[t * CH + cl];
            F2 B[H];
            Operands<T, NS>::get(sbc + t * 2 * NP + 2 * n0, B, C);
#pragma unroll
            for (int i = 0; i < H; ++i) {
                e[i] = decay2<T>(mul2(pack(d.x, d.x), ra[i]));
                u[i] = mul2(pack(d.y, d.y), B[i]);
            }
        };
        constexpr int GROUPS = TT / G, UNROLL = sizeof(T) == 2 ? GROUPS : 1;
        F2 e[G][H], u[G][H], C[G][H];
        float sum[UNROLL][G / W];                            // this lane's tokens of every group
        auto keep = [&](int g, const float * v) {
            if (lane < W) {
#pragma unroll
                for (int k = 0; k < G / W; ++k) sy[(g * G + lane * (G / W) + k) * CH + cl] = v[k];
            }
        };
#pragma unroll
        for (int k = 0; k < G; ++k) prepare(k, e[k], u[k], C[k]);
#pragma unroll UNROLL
        for (int g = 0; g < GROUPS; ++g) {
            float p[G];
#pragma unroll
            for (int k = 0; k < G; ++k) {
                F2 acc;
#pragma unroll
                for (int i = 0; i < H; ++i) {
                    s[i] = next2<T>(e[k][i], s[i], u[k][i]);
                    acc = i == 0 ? mul2(s[i], C[k][i]) : fma2(s[i], C[k][i], acc);
                }
                const float2 y = unpack(acc);
                p[k] = y.x + y.y;
                if (g + 1 < GROUPS) prepare((g + 1) * G + k, e[k], u[k], C[k]);
            }
            meet<L>(p, lane);
            if (UNROLL == 1) {
                keep(g, p);
            } else {                                         // stored at the end: no store between the loads of shared memory
#pragma unroll
                for (int k = 0; k < G / W; ++k) sum[g % UNROLL][k] = p[k];
            }
        }
        if (UNROLL > 1) {
#pragma unroll
            for (int g = 0; g < UNROLL; ++g) keep(g, sum[g]);
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < S::RX; ++i) {
            const int q = threadIdx.x + i * NT, t = q / (CH / 4);
            if (q >= S::QX || t >= m || c0 + cq >= a.ch) continue;
            const float4 y = *(const float4 *) (sy + t * CH + cq), x = cur.x[i].get(), z = cur.z[i].get();
            Quad<T>::store((T *) a.y + (size_t) (q0 + t0 + t) * a.ldy + c0 + cq,
                           make_float4((y.x + skip.x * x.x) * silu<T>(z.x) * a.out_scale, (y.y + skip.y * x.y) * silu<T>(z.y) * a.out_scale,
                                       (y.z + skip.z * x.z) * silu<T>(z.z) * a.out_scale, (y.w + skip.w * x.w) * silu<T>(z.w) * a.out_scale));
        }
        cur = nxt;
    }
    if (live && slot >= 0) {
        float v[NS];
#pragma unroll
        for (int i = 0; i < H; ++i) {
            const float2 x = unpack(s[i]);
            v[2 * i] = x.x;
            v[2 * i + 1] = x.y;
        }
        store_n<NS>(st, v);
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

template <typename T, int NS, int L>
int step(const jib_scan & a, cudaStream_t s) {
    constexpr int CH = NT / L, U = sizeof(T) == 2 && NS == 4 ? 4 : 1;
    const unsigned gx = (a.ch + CH - 1) / CH;
    if (U > 1 && a.T * gx > 148 * 8) JIB_LAUNCH((scan_step_kernel<T, NS, L, U>), dim3(gx, (a.T + U - 1) / U), NT, 0, s, a);
    else JIB_LAUNCH((scan_step_kernel<T, NS, L, 1>), dim3(gx, a.T), NT, 0, s, a);
    return launched();
}
template <typename T, int NS, int L>
int portions(const jib_scan & a, cudaStream_t s) {
    constexpr int CH = NT / L, SMEM = Scan<T, NS, L>::SMEM;
    static_assert(SMEM <= 48 * 1024, "fits without an attribute");
    JIB_LAUNCH((scan_portions_kernel<T, NS, L>), dim3((a.ch + CH - 1) / CH, a.n_seqs), NT, SMEM, s, a);
    return launched();
}

template <typename T>
int dispatch(const jib_scan & a, int single, cudaStream_t s) {
    if (a.N <= 8) return single ? step<T, 4, 2>(a, s) : portions<T, 2, 4>(a, s);
    if (a.N <= 16) return single ? step<T, 4, 4>(a, s) : portions<T, 2, 8>(a, s);
    if (a.N <= 32) return single ? step<T, 4, 8>(a, s) : portions<T, 4, 8>(a, s);
    if (a.N <= 64) return single ? step<T, 4, 16>(a, s) : portions<T, 4, 16>(a, s);
    if (a.N <= 128) return single ? step<T, 4, 32>(a, s) : portions<T, 4, 32>(a, s);
    return single ? step<T, 8, 32>(a, s) : portions<T, 8, 32>(a, s);
}

}  // namespace

extern "C" JIB_EXPORT int jib_selective_scan(const jib_scan * m, int single, int f32, void * stream) {
    const jib_scan & a = *m;
    if (a.T <= 0 || a.n_seqs <= 0) return 0;
    if (a.ch < 8 || a.ch % 8 || a.N < 8 || a.N % 8 || a.N > 256 || a.T > 65535 || a.n_seqs > 65535 || (single && a.T != a.n_seqs)) return JIB_E_ARG;
    const uintptr_t mask = f32 ? 15 : 7;                     // quads of activations, 16 bytes of fp32
    if ((((uintptr_t) a.x | (uintptr_t) a.z | (uintptr_t) a.bc | (uintptr_t) a.dt | (uintptr_t) a.y) & mask) || ((a.ldx | a.ldz | a.ldbc | a.ldy | a.lddt) & 3) ||
        (((uintptr_t) a.dt_bias | (uintptr_t) a.neg_a | (uintptr_t) a.skip | (uintptr_t) a.state) & 15))
        return JIB_E_ALIGN;
    cudaStream_t s = (cudaStream_t) stream;
    return f32 ? dispatch<float>(a, single, s) : dispatch<bf16>(a, single, s);
}
