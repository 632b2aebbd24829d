// Selective scan: every channel c carries N states with a decay of their own,
//
//   S[c][n] <- exp(dt_c a[c][n]) S[c][n] + dt_c x_c B_n;   y_c = (sum_n S[c][n] C_n + skip_c x_c) * silu(z_c) * out_scale
//
// with dt = softplus(dt_c) and B, C shared by the channels.  L lanes of a warp share a channel, NS states each.
//
//   scan_step      one token per sequence: the state is read and written once
//   scan_portions  ranges of any length: a CTA owns 128 / L channels of one sequence, keeps their states in registers and walks the
//                  tokens in tiles of TT, the next tile's inputs on their way while one is worked on
//
// The exponentials do not depend on the state, so a token costs its lane one multiply-add of latency.  The lanes' partial sums of
// several tokens meet in one butterfly that leaves each lane with one token's sum.
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
template <typename T> __device__ __forceinline__ float rate(float neg_a);            // what decay() takes
template <> __device__ __forceinline__ float rate<bf16>(float neg_a) { return neg_a * 1.4426950408889634f; }
template <> __device__ __forceinline__ float rate<float>(float neg_a) { return neg_a; }
template <typename T> __device__ __forceinline__ float decay(float v);
template <> __device__ __forceinline__ float decay<bf16>(float v) {
    float r;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(r) : "f"(v));
    return r;
}
template <> __device__ __forceinline__ float decay<float>(float v) { return expf(v); }
__device__ __forceinline__ float softplus(float v) { return fmaxf(v, 0.f) + log1pf(expf(-fabsf(v))); }

// 4 adjacent elements, kept as stored until they are needed (many loads in flight)
template <typename T> struct Quad;
template <> struct Quad<float> {
    float4 r;
    __device__ __forceinline__ void zero() { r = make_float4(0.f, 0.f, 0.f, 0.f); }
    __device__ __forceinline__ void load(const float * p) { r = *(const float4 *) p; }
    __device__ __forceinline__ float4 get() const { return r; }
    __device__ __forceinline__ static void store(float * p, float4 v) { *(float4 *) p = v; }
};
template <> struct Quad<bf16> {
    uint2 r;
    __device__ __forceinline__ void zero() { r = make_uint2(0, 0); }
    __device__ __forceinline__ void load(const bf16 * p) { r = *(const uint2 *) p; }
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
// NS adjacent floats
template <int NS> __device__ __forceinline__ void load_n(const float * p, float (&v)[NS]) {
#pragma unroll
    for (int i = 0; i < NS; i += (NS >= 4 ? 4 : 2)) {
        if (NS >= 4) {
            const float4 x = *(const float4 *) (p + i);
            v[i] = x.x; v[i + 1] = x.y; v[(i + 2) % NS] = x.z; v[(i + 3) % NS] = x.w;
        } else {
            const float2 x = *(const float2 *) (p + i);
            v[i] = x.x; v[i + 1] = x.y;
        }
    }
}
template <int NS> __device__ __forceinline__ void store_n(float * p, const float (&v)[NS]) {
#pragma unroll
    for (int i = 0; i < NS; i += (NS >= 4 ? 4 : 2)) {
        if (NS >= 4) *(float4 *) (p + i) = make_float4(v[i], v[i + 1], v[(i + 2) % NS], v[(i + 3) % NS]);
        else *(float2 *) (p + i) = make_float2(v[i], v[i + 1]);
    }
}

__device__ __forceinline__ int checked_slot(const jib_scan & a, int b, int site) {
    const int slot = a.seq_slots[b];
    if (slot >= a.n_state) {
        if (threadIdx.x == 0) jib_report(a.status, JIB_ERR_BOUNDS, site, slot);
        return -1;
    }
    return slot;
}

// ---- single tokens: grid (ceil(ch / (NT / L)), T), row t belongs to sequence t -----------------------------------------------------
template <typename T, int NS, int L>
__global__ void __launch_bounds__(NT) scan_step_kernel(const __grid_constant__ jib_scan a) {
    PDL_TRIGGER_TOP();
    const int lane = threadIdx.x % L, c = blockIdx.x * (NT / L) + threadIdx.x / L, t = blockIdx.y, n0 = lane * NS;
    const bool mine = c < a.ch, live = mine && n0 < a.N;
    const int cc = mine ? c : a.ch - 1, nn = n0 < a.N ? n0 : 0;
    float ra[NS], s[NS];
    load_n<NS>(a.neg_a + (size_t) cc * a.N + nn, ra);        // launch-invariant
    const float skip = a.skip[cc];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int slot = checked_slot(a, t, 51);
    float * st = a.state + ((size_t) (slot < 0 ? 0 : slot) * a.ch + cc) * a.N + nn;
    const bool past = slot >= 0 && live && a.positions[t] > 0;
#pragma unroll
    for (int i = 0; i < NS; ++i) s[i] = 0.f;
    if (past) load_n<NS>(st, s);
    const T * bc = (const T *) a.bc + (size_t) t * a.ldbc + nn;
    float B[NS], C[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        B[i] = to_f(bc[i]);
        C[i] = to_f(bc[a.N + i]);
    }
    const float x = to_f(((const T *) a.x)[(size_t) t * a.ldx + cc]), z = to_f(((const T *) a.z)[(size_t) t * a.ldz + cc]);
    const float dt = softplus(a.dt[(size_t) t * a.lddt + cc]), dx = dt * x;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        s[i] = decay<T>(dt * rate<T>(ra[i])) * s[i] + dx * B[i];
        y += s[i] * C[i];
    }
    if (!live) y = 0.f;
    if (live && slot >= 0) store_n<NS>(st, s);
#pragma unroll
    for (int o = L / 2; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (lane == 0 && mine) put((T *) a.y + (size_t) t * a.ldy + c, (y + skip * x) * silu<T>(z) * a.out_scale);
}

// ---- portions: grid (ceil(ch / CH), n_seqs) ----------------------------------------------------------------------------------------
template <typename T, int NS, int L>
struct Scan {
    static constexpr int NP = NS * L, CH = NT / L;
    static constexpr int TT = NP <= 64 ? 32 : 8;             // tokens of a tile
    static constexpr int GT = L < 8 ? L : 8;                 // tokens whose sums meet in one butterfly
    static constexpr int QX = TT * CH / 4, QB = TT * 2 * NP / 4;                     // quads of a tile: per channel input, of B | C
    static constexpr int RX = (QX + NT - 1) / NT, RB = (QB + NT - 1) / NT;
    static constexpr int SMEM = 4 * (TT * CH * 2 + TT * 2 * NP + TT * CH);
    Quad<T> x[RX], z[RX], bc[RB];
    Quad<float> dt[RX];
    // tokens t0 .. of the sequence's n, whose first row is q0
    __device__ __forceinline__ void load(const jib_scan & a, int q0, int n, int t0, int c0) {
#pragma unroll
        for (int i = 0; i < RX; ++i) {
            const int q = threadIdx.x + i * NT, t = t0 + q / (CH / 4), c = c0 + q % (CH / 4) * 4;
            x[i].zero(); z[i].zero(); dt[i].zero();
            if (q < QX && t < n && c < a.ch) {
                const size_t r = q0 + t;
                x[i].load((const T *) a.x + r * a.ldx + c);
                z[i].load((const T *) a.z + r * a.ldz + c);
                dt[i].load(a.dt + r * a.lddt + c);
            }
        }
        const int n4 = a.N / 2;                              // quads of a row of B | C
#pragma unroll
        for (int i = 0; i < RB; ++i) {
            const int q = threadIdx.x + i * NT, k = q / n4, t = t0 + k;
            bc[i].zero();
            if (k < TT && t < n) bc[i].load((const T *) a.bc + (size_t) (q0 + t) * a.ldbc + (q - k * n4) * 4);
        }
    }
};

template <typename T, int NS, int L>
__global__ void __launch_bounds__(NT) scan_portions_kernel(const __grid_constant__ jib_scan a) {
    using S = Scan<T, NS, L>;
    constexpr int NP = S::NP, CH = S::CH, TT = S::TT, GT = S::GT;
    extern __shared__ __align__(16) float smem[];
    float2 * sdx = (float2 *) smem;                          // [TT][CH]: step size, step size * x
    float * sb = smem + TT * CH * 2, * sc = sb + TT * NP, * sy = sc + TT * NP;       // [TT][NP], [TT][NP], [TT][CH]
    PDL_TRIGGER_TOP();
    const int lane = threadIdx.x % L, cl = threadIdx.x / L, c0 = blockIdx.x * CH, c = c0 + cl, b = blockIdx.y, n0 = lane * NS;
    const bool live = c < a.ch && n0 < a.N;
    float ra[NS], s[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) ra[i] = s[i] = 0.f;
    if (live) load_n<NS>(a.neg_a + (size_t) c * a.N + n0, ra);
#pragma unroll
    for (int i = 0; i < NS; ++i) ra[i] = rate<T>(ra[i]);
    for (int i = threadIdx.x; i < TT * 2 * NP; i += NT) sb[i] = 0.f;                 // columns past N stay zero
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int q0 = a.q_start[b], n = a.q_start[b + 1] - q0;
    if (n <= 0) return;
    S cur, nxt;
    cur.load(a, q0, n, 0, c0);
    const int slot = checked_slot(a, b, 52);
    float * st = a.state + ((size_t) (slot < 0 ? 0 : slot) * a.ch + c) * a.N + n0;
    if (live && slot >= 0 && a.positions[q0] > 0) load_n<NS>(st, s);
    __syncthreads();
    for (int t0 = 0; t0 < n; t0 += TT) {
#pragma unroll
        for (int i = 0; i < S::RX; ++i) {
            const int q = threadIdx.x + i * NT, t = q / (CH / 4);
            if (q >= S::QX) continue;
            const float4 x = cur.x[i].get(), d = cur.dt[i].get();
            const bool in = t0 + t < n;                      // past the end: the state passes through
            const float dt[4] = {softplus(d.x), softplus(d.y), softplus(d.z), softplus(d.w)};
            float4 * o = (float4 *) (sdx + t * CH + q % (CH / 4) * 4);
            o[0] = in ? make_float4(dt[0], dt[0] * x.x, dt[1], dt[1] * x.y) : make_float4(0.f, 0.f, 0.f, 0.f);
            o[1] = in ? make_float4(dt[2], dt[2] * x.z, dt[3], dt[3] * x.w) : make_float4(0.f, 0.f, 0.f, 0.f);
        }
        const int n4 = a.N / 2;
#pragma unroll
        for (int i = 0; i < S::RB; ++i) {
            const int q = threadIdx.x + i * NT, t = q / n4, col = (q - t * n4) * 4;
            if (t < TT) *(float4 *) ((col < a.N ? sb + col : sc + col - a.N) + t * NP) = cur.bc[i].get();
        }
        __syncthreads();
        if (t0 + TT < n) nxt.load(a, q0, n, t0 + TT, c0);
        const int m = min(TT, n - t0);
#pragma unroll 1
        for (int g = 0; g < m; g += GT) {
            float p[GT];
#pragma unroll
            for (int k = 0; k < GT; ++k) {
                const float2 d = sdx[(g + k) * CH + cl];
                float B[NS], C[NS];
                load_n<NS>(sb + (g + k) * NP + n0, B);
                load_n<NS>(sc + (g + k) * NP + n0, C);
                p[k] = 0.f;
#pragma unroll
                for (int i = 0; i < NS; ++i) {
                    s[i] = decay<T>(d.x * ra[i]) * s[i] + d.y * B[i];
                    p[k] += s[i] * C[i];
                }
            }
#pragma unroll
            for (int o = GT / 2; o > 0; o >>= 1)
#pragma unroll
                for (int k = 0; k < o; ++k) {
                    const bool up = (lane & o) != 0;
                    const float keep = up ? p[k + o] : p[k], send = up ? p[k] : p[k + o];
                    p[k] = keep + __shfl_xor_sync(0xffffffffu, send, o);
                }
#pragma unroll
            for (int o = GT; o < L; o <<= 1) p[0] += __shfl_xor_sync(0xffffffffu, p[0], o);
            if (lane < GT) sy[(g + lane) * CH + cl] = p[0];
        }
        __syncthreads();
#pragma unroll
        for (int i = 0; i < S::RX; ++i) {
            const int q = threadIdx.x + i * NT, t = q / (CH / 4), cq = q % (CH / 4) * 4;
            if (q >= S::QX || t >= m || c0 + cq >= a.ch) continue;
            const float4 y = *(const float4 *) (sy + t * CH + cq), x = cur.x[i].get(), z = cur.z[i].get(), k = *(const float4 *) (a.skip + c0 + cq);
            Quad<T>::store((T *) a.y + (size_t) (q0 + t0 + t) * a.ldy + c0 + cq,
                           make_float4((y.x + k.x * x.x) * silu<T>(z.x) * a.out_scale, (y.y + k.y * x.y) * silu<T>(z.y) * a.out_scale,
                                       (y.z + k.z * x.z) * silu<T>(z.z) * a.out_scale, (y.w + k.w * x.w) * silu<T>(z.w) * a.out_scale));
        }
        cur = nxt;
    }
    if (live && slot >= 0) store_n<NS>(st, s);
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

template <typename T, int NS, int L>
int run(const jib_scan & a, int single, cudaStream_t s) {
    constexpr int CH = NT / L;
    if (single) {
        JIB_LAUNCH((scan_step_kernel<T, NS, L>), dim3((a.ch + CH - 1) / CH, a.T), NT, 0, s, a);
        return launched();
    }
    constexpr int SMEM = Scan<T, NS, L>::SMEM;
    static_assert(SMEM <= 48 * 1024, "fits without an attribute");
    JIB_LAUNCH((scan_portions_kernel<T, NS, L>), dim3((a.ch + CH - 1) / CH, a.n_seqs), NT, SMEM, s, a);
    return launched();
}

template <typename T>
int dispatch(const jib_scan & a, int single, cudaStream_t s) {
    if (a.N <= 8) return run<T, 2, 4>(a, single, s);
    if (a.N <= 16) return run<T, 2, 8>(a, single, s);
    if (a.N <= 32) return run<T, 4, 8>(a, single, s);
    if (a.N <= 64) return run<T, 4, 16>(a, single, s);
    if (a.N <= 128) return run<T, 4, 32>(a, single, s);
    return run<T, 8, 32>(a, single, s);
}

}  // namespace

extern "C" JIB_EXPORT int jib_selective_scan(const jib_scan * m, int single, int f32, void * stream) {
    const jib_scan & a = *m;
    if (a.T <= 0 || a.n_seqs <= 0) return 0;
    if (a.ch < 8 || a.ch % 8 || a.N < 8 || a.N % 8 || a.N > 256 || a.T > 65535 || a.n_seqs > 65535 || (single && a.T != a.n_seqs)) return JIB_E_ARG;
    const uintptr_t mask = f32 ? 15 : 7;                     // quads of activations, 16 bytes of fp32
    if ((((uintptr_t) a.x | (uintptr_t) a.z | (uintptr_t) a.bc | (uintptr_t) a.y) & mask) || ((a.ldx | a.ldz | a.ldbc | a.ldy | a.lddt) & 3) ||
        (((uintptr_t) a.dt | (uintptr_t) a.neg_a | (uintptr_t) a.skip | (uintptr_t) a.state) & 15))
        return JIB_E_ALIGN;
    cudaStream_t s = (cudaStream_t) stream;
    return f32 ? dispatch<float>(a, single, s) : dispatch<bf16>(a, single, s);
}
