// Portions through the matrix-state mixers on tensor cores (bf16 activations, K of 64 or 128, V a multiple of 16).
//
// Within a chunk of 32 tokens, with G_t the running sum of the log decays (G_t <= 0) and S the state before the chunk:
//
//   o_t = S^T (q_t e^{G_t}) + sum_{s <= t} A_ts u_s         A_ts = sum_c q_tc k_sc e^{G_tc - G_sc}
//   S'  = e^{G_C} S + sum_s (k_s e^{G_C - G_s}) u_s^T
//   DELTA: u = b (v - .) is the solution of a triangular system, (1 + b B) u = b (v - S^T (k e^{G})) with B_ts = sum_c k_tc k_sc e^{G_tc - G_sc},
//   s < t:  u = U0 - W S with W = (1 + b B)^-1 b (k e^{G}), U0 = (1 + b B)^-1 b v.
//
// Every exponent that occurs is a difference G_t - G_s with s <= t and so at most 0, however fast the decay: nothing overflows and no
// quotient of vanishing products is formed.
//   prepare (one CTA per chunk and head; SSD: per chunk and group): convolution, unit norm, decays, A, W, U0.  Independent of S.
//   pass    (one CTA per head and 16 value columns, SSD 32): walks the chunks, S in registers, everything else a product of small matrices.
// State, decays, A, W, U0 are fp32; the tensor cores see each as a sum of two bf16 numbers and the products hi * hi + hi * lo + lo * hi
// (about 16 bits of mantissa); q and k of SSD are bf16 to begin with.  Accumulation is fp32.
#include "pdl.cuh"
#include "state_mix.cuh"

namespace {

using namespace state_mix;

constexpr int C = 32, VB = 16, NT = 256, STAGES = 3;
constexpr float LOG2E = 1.4426950408889634f;
constexpr int QK_LD = 32;                                    // row stride of SSD's q . k table (fp32)

// A chunk's record: bf16 tiles of 32 rows x K columns in 16-byte units u of row r stored at u ^ (r & 7); A: 32 x 32, unit u ^ (r / 2 & 3).
template <int KIND, int K> struct Rec {
    static constexpr int TILE = C * K * 2, ATILE = C * C * 2;
    static constexpr int Q = 0, D = KIND == SSD ? TILE : 2 * TILE;                        // q e^G, k e^{G_C - G} (SSD: q, k)
    static constexpr int A = KIND == SSD ? 2 * TILE : 4 * TILE;                           // hi, lo (SSD: q . k fp32)
    static constexpr int W = A + 2 * ATILE;                                               // DELTA
    static constexpr int E = W + (KIND == DELTA ? 2 * TILE : 0);                          // e^{G_C}
    static constexpr int BYTES = KIND == SSD ? A + C * QK_LD * 4 : E + K * 4;
};

// run index: sequence b's chunks start at q_start[b] / C + b; indices in the gaps have no tokens
__device__ __forceinline__ int chunk_key(const int * q_start, int b) { return q_start[b] / C + b; }
__device__ __forceinline__ int chunk_seq(const jib_state_mix & a, int ci) {
    int b = 0, hi = a.n_seqs;
    while (hi - b > 1) {
        const int mid = (b + hi) >> 1;
        if (chunk_key(a.q_start, mid) <= ci) b = mid; else hi = mid;
    }
    return b;
}

__device__ __forceinline__ void load4(const bf16 * p, float (&v)[4]) {
    const uint2 r = *(const uint2 *) p;
    const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *) &r.x), y = __bfloat1622float2(*(const __nv_bfloat162 *) &r.y);
    v[0] = x.x; v[1] = x.y; v[2] = y.x; v[3] = y.y;
}
// Two fp32 operations per instruction.
struct F2 { unsigned long long v; };
__device__ __forceinline__ F2 f2(float x, float y) {
    F2 r;
    asm("mov.b64 %0, {%1, %2};" : "=l"(r.v) : "f"(x), "f"(y));
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
__device__ __forceinline__ float sum2(F2 a) {
    const float2 x = unpack(a);
    return x.x + x.y;
}
// 4 columns from column c on of tokens i0 .. i0 + 7 of a range (its first token: row q0, position p0; n tokens): convolved and silu'd.
// Up to 4 taps; every row is loaded once, all loads in flight together.  Rows past the range are zero.
__device__ __forceinline__ void conv_run(const jib_state_mix & a, int q0, int p0, int n, int i0, int c, int slot, float (&out)[8][4]) {
    const bf16 * x = (const bf16 *) a.proj + (size_t) q0 * a.ld + c;
    float v[11][4];
#pragma unroll
    for (int r = 0; r < 11; ++r) {
        const int i = i0 + r - 3;
#pragma unroll
        for (int e = 0; e < 4; ++e) v[r][e] = 0.f;
        if (r < 3 && 3 - r >= a.taps) continue;              // further back than the filter reaches
        if (i >= 0 && i < n) load4(x + (long long) i * a.ld, v[r]);
        else if (i < 0 && slot >= 0 && p0 + i >= 0)
            load4((const bf16 *) a.conv_state + ((size_t) slot * a.taps + (p0 + i) % a.taps) * a.n_conv + c - a.conv0, v[r]);
    }
    if (a.taps == 0) {
#pragma unroll
        for (int r = 0; r < 8; ++r)
#pragma unroll
            for (int e = 0; e < 4; ++e) out[r][e] = v[r + 3][e];
        return;
    }
    float4 w[4], b = make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
    for (int j = 0; j < 4; ++j) {
        w[j] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (j >= 4 - a.taps) w[j] = *(const float4 *) (a.conv_w + (size_t) (j - (4 - a.taps)) * a.n_conv + c - a.conv0);
    }
    if (a.conv_b != nullptr) b = *(const float4 *) (a.conv_b + c - a.conv0);
#pragma unroll
    for (int r = 0; r < 8; ++r) {
        F2 s0 = f2(b.x, b.y), s1 = f2(b.z, b.w);
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            s0 = fma2(f2(w[j].x, w[j].y), f2(v[r + j][0], v[r + j][1]), s0);
            s1 = fma2(f2(w[j].z, w[j].w), f2(v[r + j][2], v[r + j][3]), s1);
        }
        const float2 a0 = unpack(s0), a1 = unpack(s1);
        const float acc[4] = {a0.x, a0.y, a1.x, a1.y};
#pragma unroll
        for (int e = 0; e < 4; ++e) out[r][e] = i0 + r < n ? silu<bf16>(acc[e]) : 0.f;
    }
}

__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
// log(1 + e^x) to a few ulp: max(x, 0) + log(1 + y) with y = e^-|x|, and log(1 + y) = 2 atanh(t), t = y / (2 + y) <= 1 / 3, by its
// power series.
__device__ __forceinline__ float softplus_series(float x) {
    const float y = ex2(-fabsf(x) * LOG2E), t = __fdividef(y, 2.f + y), z = t * t;
    float s = 1.f / 15.f;
    s = s * z + 1.f / 13.f;
    s = s * z + 1.f / 11.f;
    s = s * z + 1.f / 9.f;
    s = s * z + 1.f / 7.f;
    s = s * z + 1.f / 5.f;
    s = s * z + 1.f / 3.f;
    s = s * z + 1.f;
    return fmaxf(x, 0.f) + 2.f * t * s;
}
// x = hi + lo, both bf16; two numbers packed
__device__ __forceinline__ void split2(float x, float y, uint32_t & hi, uint32_t & lo) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    const float2 f = __bfloat1622float2(h);
    const __nv_bfloat162 l = __floats2bfloat162_rn(x - f.x, y - f.y);
    hi = *(const uint32_t *) &h;
    lo = *(const uint32_t *) &l;
}
template <int K> __device__ __forceinline__ int tile_off(int r, int c) { return r * (K * 2) + (((c >> 3) ^ (r & 7)) << 4) + (c & 7) * 2; }
__device__ __forceinline__ int a_off(int r, int c) { return r * 64 + (((c >> 3) ^ ((r >> 1) & 3)) << 4) + (c & 7) * 2; }
template <int K> __device__ __forceinline__ void put_tile4(uint8_t * hi, int r, int c, float4 v) {
    uint2 h, l;
    split2(v.x, v.y, h.x, l.x);
    split2(v.z, v.w, h.y, l.y);
    *(uint2 *) (hi + tile_off<K>(r, c)) = h;
    *(uint2 *) (hi + C * K * 2 + tile_off<K>(r, c)) = l;
}

// ---- prepare: DELTA, LINEAR ------------------------------------------------------------------------------------------------------
template <int K> constexpr int prep_smem(int V) { return 4 * (3 * C * (K + 4) + C * (V + 4) + C * 36 + 3 * C); }

template <int KIND, int K>
__global__ void __launch_bounds__(NT, 3) chunk_prepare_kernel(const __grid_constant__ jib_state_mix a) {
    using R = Rec<KIND, K>;
    constexpr int KS = K + 4;
    extern __shared__ __align__(16) float sm[];
    PDL_TRIGGER_TOP();
    const int V = a.V, VS = V + 4, tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    float * q = sm, * k = q + C * KS, * G = k + C * KS, * v = G + C * KS, * B = v + C * VS, * beta = B + C * 36, * norm = beta + C;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int ci = blockIdx.x, h = blockIdx.y, b = chunk_seq(a, ci);
    const int r0 = a.q_start[b], nr = a.q_start[b + 1] - r0, t0 = (ci - chunk_key(a.q_start, b)) * C;
    if (t0 < 0 || t0 >= nr) return;
    const int p0 = a.positions[r0], n = min(C, nr - t0);
    const int slot = a.taps > 0 ? checked_slot(a, b, 45) : -1;
    // inputs: 8 tokens x 4 columns per job
    const int jk = K / 4 * (C / 8), jv = V / 4 * (C / 8);
    for (int j = tid; j < 3 * jk + jv; j += NT) {
        float x[8][4];
        float * dst;
        int ld, col, run;
        if (j < 2 * jk + jv) {
            const int jj = j < jk ? j : j < 2 * jk ? j - jk : j - 2 * jk, w = j < 2 * jk ? K / 4 : V / 4;
            col = jj % w * 4;
            run = jj / w * 8;
            ld = j < 2 * jk ? KS : VS;
            dst = j < jk ? q : j < 2 * jk ? k : v;
            conv_run(a, r0, p0, nr, t0 + run, (j < jk ? a.q_off + h / a.rep * K : j < 2 * jk ? a.k_off + h / a.rep * K : a.v_off + h * V) + col, slot, x);
        } else {
            const int jj = j - 2 * jk - jv;
            col = jj % (K / 4) * 4;
            run = jj / (K / 4) * 8;
            ld = KS;
            dst = G;
            const bf16 * z = (const bf16 *) a.dec_in + (size_t) (r0 + t0) * a.ld_dec + h * K + col;
            const float4 bias = *(const float4 *) (a.bias + h * K + col);
            const float f = LOG2E * (KIND == DELTA ? a.neg_a[h] : -a.inv_tau);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
#pragma unroll
                for (int e = 0; e < 4; ++e) x[r][e] = 0.f;
                if (run + r < n) load4(z + (size_t) (run + r) * a.ld_dec, x[r]);
            }
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                const float s = KIND == DELTA ? 1.f : -1.f;
                x[r][0] = run + r < n ? f * softplus_series(s * (x[r][0] + bias.x)) : 0.f;
                x[r][1] = run + r < n ? f * softplus_series(s * (x[r][1] + bias.y)) : 0.f;
                x[r][2] = run + r < n ? f * softplus_series(s * (x[r][2] + bias.z)) : 0.f;
                x[r][3] = run + r < n ? f * softplus_series(s * (x[r][3] + bias.w)) : 0.f;
            }
        }
#pragma unroll
        for (int r = 0; r < 8; ++r) *(float4 *) (dst + (run + r) * ld + col) = make_float4(x[r][0], x[r][1], x[r][2], x[r][3]);
    }
    if (KIND == DELTA && tid < C)
        beta[tid] = tid < n ? head_factor<DELTA>(a, to_f(((const bf16 *) a.proj)[(size_t) (r0 + t0 + tid) * a.ld + a.s_off + h]), h) : 0.f;
    __syncthreads();
    // unit norms (folded into q and k) and running sums of the log decays
    if (KIND == DELTA) {
        for (int r = warp; r < 2 * C; r += NT / 32) {
            const float * x = (r < C ? q : k) + (r & (C - 1)) * KS;
            float ss = 0.f;
            for (int c = lane; c < K; c += 32) ss += x[c] * x[c];
            ss = warp_sum(ss);
            if (lane == 0) norm[r] = rsqrtf(ss + 1e-6f) * (r < C ? a.q_scale : 1.f);
        }
    } else if (tid < 2 * C) {
        norm[tid] = tid < C ? a.q_scale : 1.f;
    }
    for (int c = tid; c < K; c += NT) {
        float g[C], s = 0.f;
#pragma unroll
        for (int t = 0; t < C; ++t) g[t] = G[t * KS + c];
#pragma unroll
        for (int t = 0; t < C; ++t) {
            s += g[t];
            G[t * KS + c] = s;
        }
    }
    __syncthreads();
    for (int i = tid; i < 2 * C * (K / 4); i += NT) {
        const int r = i / (K / 4), c = i % (K / 4) * 4;
        float4 * x = (float4 *) ((r < C ? q : k) + (r & (C - 1)) * KS + c);
        const float s = norm[r];
        float4 y = *x;
        y.x *= s; y.y *= s; y.z *= s; y.w *= s;
        *x = y;
    }
    __syncthreads();
    uint8_t * rec = (uint8_t *) a.chunk + ((size_t) ci * a.H + h) * (R::BYTES + C * 4 * V);
    // A and B: one thread per pair s < t (rows i and C - 1 - i together have C - 1 of them)
    for (int i = tid; i < C * (C - 1) / 2; i += NT) {
        const int i1 = i / (C - 1), j = i % (C - 1);
        const int t = j < i1 ? i1 : C - 1 - i1, s = j < i1 ? j : j - i1;
        const float * qt = q + t * KS, * kt = k + t * KS, * gt = G + t * KS, * ks = k + s * KS, * gs = G + s * KS;
        F2 q0 = f2(0.f, 0.f), q1 = q0, k0 = q0, k1 = q0;
        const F2 minus = f2(-1.f, -1.f);
#pragma unroll 4
        for (int c = 0; c < K; c += 4) {
            const float4 x = *(const float4 *) (gt + c), y = *(const float4 *) (gs + c), z = *(const float4 *) (ks + c), u = *(const float4 *) (qt + c);
            const float2 d0 = unpack(fma2(f2(y.x, y.y), minus, f2(x.x, x.y))), d1 = unpack(fma2(f2(y.z, y.w), minus, f2(x.z, x.w)));
            const F2 e0 = mul2(f2(z.x, z.y), f2(ex2(d0.x), ex2(d0.y))), e1 = mul2(f2(z.z, z.w), f2(ex2(d1.x), ex2(d1.y)));
            q0 = fma2(f2(u.x, u.y), e0, q0);
            q1 = fma2(f2(u.z, u.w), e1, q1);
            if (KIND == DELTA) {
                const float4 w = *(const float4 *) (kt + c);
                k0 = fma2(f2(w.x, w.y), e0, k0);
                k1 = fma2(f2(w.z, w.w), e1, k1);
            }
        }
        const float aq = sum2(q0) + sum2(q1), ak = sum2(k0) + sum2(k1);
        if (KIND == DELTA) {
            B[t * 36 + s] = ak * beta[t];
            B[s * 36 + t] = 0.f;
        }
        const bf16 hi = __float2bfloat16(aq);
        *(bf16 *) (rec + R::A + a_off(t, s)) = hi;
        *(bf16 *) (rec + R::A + R::ATILE + a_off(t, s)) = __float2bfloat16(aq - to_f(hi));
        *(bf16 *) (rec + R::A + a_off(s, t)) = __float2bfloat16(0.f);
        *(bf16 *) (rec + R::A + R::ATILE + a_off(s, t)) = __float2bfloat16(0.f);
    }
    for (int t = warp; t < C; t += NT / 32) {                // the diagonal
        float d = 0.f;
        for (int c = lane; c < K; c += 32) d += q[t * KS + c] * k[t * KS + c];
        d = warp_sum(d);
        if (lane == 0) {
            const bf16 hi = __float2bfloat16(d);
            *(bf16 *) (rec + R::A + a_off(t, t)) = hi;
            *(bf16 *) (rec + R::A + R::ATILE + a_off(t, t)) = __float2bfloat16(d - to_f(hi));
            if (KIND == DELTA) B[t * 36 + t] = 0.f;
        }
    }
    for (int i = tid; i < C * (K / 4); i += NT) {            // q e^G, k e^{G_C - G}
        const int t = i / (K / 4), c = i % (K / 4) * 4;
        const float4 g = *(const float4 *) (G + t * KS + c), e = *(const float4 *) (G + (C - 1) * KS + c);
        const float4 x = *(const float4 *) (q + t * KS + c), y = *(const float4 *) (k + t * KS + c);
        put_tile4<K>(rec + R::Q, t, c, make_float4(x.x * ex2(g.x), x.y * ex2(g.y), x.z * ex2(g.z), x.w * ex2(g.w)));
        put_tile4<K>(rec + R::D, t, c, make_float4(y.x * ex2(e.x - g.x), y.y * ex2(e.y - g.y), y.z * ex2(e.z - g.z), y.w * ex2(e.w - g.w)));
    }
    for (int c = tid; c < K; c += NT) ((float *) (rec + R::E))[c] = ex2(G[(C - 1) * KS + c]);
    float * U = (float *) (rec + R::BYTES);
    if (KIND == LINEAR) {
        for (int i = tid; i < C * V; i += NT) {
            const int t = i / V, c = i % V;
            U[(c >> 4) * (C * VB) + t * VB + (c & 15)] = v[t * VS + c];
        }
        return;
    }
    __syncthreads();
    // forward substitution, one right-hand side per thread: columns of k e^G, then of v
    for (int c = tid; c < K + V; c += NT) {
        float x[C];
#pragma unroll
        for (int t = 0; t < C; ++t) x[t] = beta[t] * (c < K ? k[t * KS + c] * ex2(G[t * KS + c]) : v[t * VS + c - K]);
#pragma unroll
        for (int t = 1; t < C; ++t) {                        // B is 0 from its diagonal on: whole vectors of 4
            F2 s0 = f2(0.f, 0.f), s1 = s0;
#pragma unroll
            for (int s = 0; s < t; s += 4) {
                const float4 w = *(const float4 *) (B + t * 36 + s);
                s0 = fma2(f2(w.x, w.y), f2(x[s], x[s + 1]), s0);
                if (s + 2 < t) s1 = fma2(f2(w.z, w.w), f2(x[s + 2], x[s + 3]), s1);
            }
            x[t] -= sum2(s0) + sum2(s1);
        }
        if (c < K) {
#pragma unroll
            for (int t = 0; t < C; ++t) {
                const bf16 hi = __float2bfloat16(x[t]);
                *(bf16 *) (rec + R::W + tile_off<K>(t, c)) = hi;
                *(bf16 *) (rec + R::W + R::TILE + tile_off<K>(t, c)) = __float2bfloat16(x[t] - to_f(hi));
            }
        } else {
            const int cc = c - K;
#pragma unroll
            for (int t = 0; t < C; ++t) U[(cc >> 4) * (C * VB) + t * VB + (cc & 15)] = x[t];
        }
    }
}

// ---- prepare: SSD ------------------------------------------------------------------------------------------------------------------
// blockIdx.y < groups: q and k tiles of a group and their products; then runs of 256 value columns (bf16 into a.v), then the factors.
template <int K>
__global__ void __launch_bounds__(NT, 3) chunk_prepare_ssd_kernel(const __grid_constant__ jib_state_mix a) {
    using R = Rec<SSD, K>;
    constexpr int KS = K + 4;
    extern __shared__ __align__(16) float sm[];
    PDL_TRIGGER_TOP();
    const int tid = threadIdx.x, groups = a.H / a.rep, inner = a.H * a.V;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int ci = blockIdx.x, b = chunk_seq(a, ci);
    const int r0 = a.q_start[b], nr = a.q_start[b + 1] - r0, t0 = (ci - chunk_key(a.q_start, b)) * C;
    if (t0 < 0 || t0 >= nr) return;
    const int p0 = a.positions[r0], n = min(C, nr - t0);
    const int slot = a.taps > 0 ? checked_slot(a, b, 45) : -1;
    int y = blockIdx.y;
    if (y < groups) {
        float * q = sm, * k = sm + C * KS;
        uint8_t * rec = (uint8_t *) a.chunk + ((size_t) ci * groups + y) * R::BYTES;
        const int jk = K / 4 * (C / 8);
        for (int j = tid; j < 2 * jk; j += NT) {
            float x[8][4];
            const int jj = j < jk ? j : j - jk, col = jj % (K / 4) * 4, run = jj / (K / 4) * 8;
            conv_run(a, r0, p0, nr, t0 + run, (j < jk ? a.q_off : a.k_off) + y * K + col, slot, x);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                __nv_bfloat162 v[2] = {__floats2bfloat162_rn(x[r][0], x[r][1]), __floats2bfloat162_rn(x[r][2], x[r][3])};
                *(uint2 *) (rec + (j < jk ? R::Q : R::D) + tile_off<K>(run + r, col)) = *(const uint2 *) v;
                const float2 f0 = __bfloat1622float2(v[0]), f1 = __bfloat1622float2(v[1]);
                *(float4 *) ((j < jk ? q : k) + (run + r) * KS + col) = make_float4(f0.x, f0.y, f1.x, f1.y);
            }
        }
        __syncthreads();
        for (int i = tid; i < C * C; i += NT) {
            const int t = i / C, s = i % C;
            if (s > t) continue;
            float d = 0.f;
#pragma unroll 4
            for (int c = 0; c < K; c += 4) {
                const float4 x = *(const float4 *) (q + t * KS + c), z = *(const float4 *) (k + s * KS + c);
                d += x.x * z.x + x.y * z.y + x.z * z.z + x.w * z.w;
            }
            ((float *) (rec + R::A))[t * QK_LD + s] = d;
        }
        return;
    }
    y -= groups;
    const int vblocks = (inner + 255) / 256;
    if (y < vblocks) {
        const int col = y * 256 + (tid & 63) * 4, run = (tid >> 6) * 8;
        if (col >= inner) return;
        float x[8][4];
        conv_run(a, r0, p0, nr, t0 + run, a.v_off + col, slot, x);
#pragma unroll
        for (int r = 0; r < 8; ++r) {
            if (run + r >= n) break;
            __nv_bfloat162 v[2] = {__floats2bfloat162_rn(x[r][0], x[r][1]), __floats2bfloat162_rn(x[r][2], x[r][3])};
            *(uint2 *) ((bf16 *) a.v + (size_t) (r0 + t0 + run + r) * inner + col) = *(const uint2 *) v;
        }
        return;
    }
    for (int i = tid; i < n * a.H; i += NT) {
        const size_t row = r0 + t0 + i / a.H;
        const int h = i % a.H;
        a.s[row * a.H + h] = head_factor<SSD>(a, to_f(((const bf16 *) a.proj)[row * a.ld + a.s_off + h]), h);
    }
}

// ---- pass --------------------------------------------------------------------------------------------------------------------------
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

constexpr int BS = VB + 8;                                   // row stride of the [.][VB] bf16 operands (48 bytes: rows hit different banks)

template <int KIND, int K> struct Pass {
    using R = Rec<KIND, K>;
    static constexpr int X = R::BYTES;                       // U0 fp32 [C][VB]
    static constexpr int STAGE = X + C * VB * 4;
    static constexpr int S = STAGES * STAGE;                 // S hi, lo [K][BS]
    static constexpr int U = S + 2 * K * BS * 2;             // U hi, lo [C][BS]
    static constexpr int SMEM = U + 2 * C * BS * 2;
};

// DELTA, LINEAR.  Warps 0 - 3 own a 16 x 8 tile of o each, warps 4 - 7 one of u; all warps own tiles of S.  Two barriers per chunk: u is
// there (and so is the next chunk's record), S is there.  Operands that depend on neither are in registers by then.
template <int KIND, int K>
__global__ void __launch_bounds__(NT, 1) chunk_pass_kernel(const __grid_constant__ jib_state_mix a) {
    using R = Rec<KIND, K>;
    using P = Pass<KIND, K>;
    constexpr int TPW = K / 64;                              // 16 x 8 tiles of S per warp (K / 16 x 2 over 8 warps), side by side
    extern __shared__ __align__(16) uint8_t smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int splits = a.V / VB, h = blockIdx.x / splits, vs = blockIdx.x % splits, b = blockIdx.y, V = a.V, H = a.H;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int r0 = a.q_start[b], n = a.q_start[b + 1] - r0;
    if (n <= 0) return;
    const int slot = checked_slot(a, b, 46);
    const int chunks = (n + C - 1) / C;
    const uint8_t * rec0 = (const uint8_t *) a.chunk + ((size_t) chunk_key(a.q_start, b) * H + h) * (R::BYTES + C * 4 * V);
    const size_t rec_step = (size_t) H * (R::BYTES + C * 4 * V);
    auto stage = [&](int i) {
        if (i < chunks) {
            uint8_t * dst = smem + i % STAGES * P::STAGE;
            const uint8_t * src = rec0 + i * rec_step;
            for (int o = tid * 16; o < R::BYTES; o += NT * 16) cp16(dst + o, src + o);
            if (tid < C * VB / 4) cp16(dst + P::X + tid * 16, src + R::BYTES + vs * (C * VB * 4) + tid * 16);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0);
    stage(1);
    store_conv_tail<bf16>(a, slot, r0, n, blockIdx.x * NT + tid, gridDim.x * NT);

    bf16 * Sh = (bf16 *) (smem + P::S), * Uh = (bf16 *) (smem + P::U);
    const uint32_t S_addr = sm100::smem_u32(Sh), U_addr = sm100::smem_u32(Uh);
    constexpr uint32_t S_LO = K * BS * 2, U_LO = C * BS * 2;
    const int fr = lane >> 2, fc = (lane & 3) * 2;           // accumulator element: rows fr, fr + 8, columns fc, fc + 1
    const int lr = lane & 15, lu = lane >> 4;                // ldmatrix lane addresses: operand rows (16 rows x 2 units) ...
    const int tr = (lane & 7) + ((lane >> 4) << 3), tu = (lane >> 3) & 1;         // ... and k^T tiles (rows = tokens)
    const int mt = (warp >> 1) & 1, nt = warp & 1;           // this warp's tile of o or u
    const bool is_o = warp < 4;
    const int sm_ = warp * TPW >> 1, sn0 = TPW == 2 ? 0 : warp & 1;               // tiles of S: rows 16 sm_, columns 8 (sn0 + i)
    float st[TPW][4];
    float * state = a.state + (((size_t) (slot < 0 ? 0 : slot) * H + h) * K + sm_ * 16 + fr) * V + vs * VB + fc;
    const bool past = slot >= 0 && a.positions[r0] > 0;
#pragma unroll
    for (int i = 0; i < TPW; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const float2 x = past ? *(const float2 *) (state + (size_t) (8 * e) * V + (sn0 + i) * 8) : make_float2(0.f, 0.f);
            st[i][2 * e] = x.x;
            st[i][2 * e + 1] = x.y;
        }
    auto publish_state = [&]() {
#pragma unroll
        for (int i = 0; i < TPW; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                uint32_t hi, lo;
                split2(st[i][2 * e], st[i][2 * e + 1], hi, lo);
                bf16 * p = Sh + (sm_ * 16 + fr + 8 * e) * BS + (sn0 + i) * 8 + fc;
                *(uint32_t *) p = hi;
                *(uint32_t *) (p + K * BS) = lo;
            }
    };
    uint32_t xh[K / 16][4], xl[K / 16][4];                   // q e^G or W rows of this warp's tile
    auto load_rows = [&](int ch) {
        if (!is_o && KIND == LINEAR) return;
        const int r = mt * 16 + lr;
        const uint32_t base = sm100::smem_u32(smem + ch % STAGES * P::STAGE) + (is_o ? R::Q : R::W) + r * (K * 2);
#pragma unroll
        for (int kk = 0; kk < K / 16; ++kk) {
            ldm4(xh[kk], base + (((kk * 2 + lu) ^ (r & 7)) << 4));
            ldm4(xl[kk], base + R::TILE + (((kk * 2 + lu) ^ (r & 7)) << 4));
        }
    };
    publish_state();
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    load_rows(0);
    for (int ch = 0; ch < chunks; ++ch) {
        stage(ch + 2);                                       // into the buffer of chunk ch - 1
        const uint8_t * rec = smem + ch % STAGES * P::STAGE;
        const uint32_t rec_addr = sm100::smem_u32(rec);
        float o[4] = {0.f, 0.f, 0.f, 0.f};
        if (is_o || KIND == DELTA) {
            float acc[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
            for (int kk = 0; kk < K / 32; ++kk) {            // 32 channels at a time
                uint32_t bh[4], bl[4];
                const uint32_t off = ((kk * 32 + lane) * BS + nt * 8) * 2;
                ldm4t(bh, S_addr + off);
                ldm4t(bl, S_addr + S_LO + off);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    mma(acc[e], xh[2 * kk + e], bh[2 * e], bh[2 * e + 1]);
                    mma(acc[2], xh[2 * kk + e], bl[2 * e], bl[2 * e + 1]);
                    mma(acc[3], xl[2 * kk + e], bh[2 * e], bh[2 * e + 1]);
                }
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) o[e] = (acc[0][e] + acc[1][e]) + (acc[2][e] + acc[3][e]);
        }
        if (!is_o) {                                         // u of this chunk as an operand
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int row = mt * 16 + fr + 8 * e, c = nt * 8 + fc;
                const float2 x = *(const float2 *) (rec + P::X + (row * VB + c) * 4);
                uint32_t hi, lo;
                split2(x.x - o[2 * e], x.y - o[2 * e + 1], hi, lo);
                bf16 * p = Uh + row * BS + c;
                *(uint32_t *) p = hi;
                *(uint32_t *) (p + C * BS) = lo;
            }
        }
        // what the second half needs of the record
        uint32_t dh[2][4], dl[2][4], ah[2][4], al[2][4];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int r = e * 16 + tr;
            const uint32_t d = rec_addr + R::D + r * (K * 2) + (((sm_ * 2 + tu) ^ (r & 7)) << 4);
            ldm4t(dh[e], d);
            ldm4t(dl[e], d + R::TILE);
            if (is_o) {
                const int q = mt * 16 + lr;
                const uint32_t p = rec_addr + R::A + q * 64 + (((e * 2 + lu) ^ ((q >> 1) & 3)) << 4);
                ldm4(ah[e], p);
                ldm4(al[e], p + R::ATILE);
            }
        }
        const float * E = (const float *) (rec + R::E) + sm_ * 16 + fr;
        const float e0 = E[0], e1 = E[8];
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();                                     // u, and the next chunk's record
        uint32_t uh[2][4], ul[2][4];                         // both 8-column units of u
#pragma unroll
        for (int i = 0; i < 2; ++i) {
            ldm4t(uh[i], U_addr + (lane * BS + i * 8) * 2);
            ldm4t(ul[i], U_addr + U_LO + (lane * BS + i * 8) * 2);
        }
        // S' = e^{G_C} S + (k e^{G_C - G})^T u
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            const int c = TPW == 2 ? i : sn0;
            float p1[4] = {0.f, 0.f, 0.f, 0.f}, p2[4] = {0.f, 0.f, 0.f, 0.f};
            st[i][0] *= e0; st[i][1] *= e0; st[i][2] *= e1; st[i][3] *= e1;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const uint32_t h0 = c ? uh[1][2 * e] : uh[0][2 * e], h1 = c ? uh[1][2 * e + 1] : uh[0][2 * e + 1];
                const uint32_t l0 = c ? ul[1][2 * e] : ul[0][2 * e], l1 = c ? ul[1][2 * e + 1] : ul[0][2 * e + 1];
                mma(st[i], dh[e], h0, h1);
                mma(p1, dh[e], l0, l1);
                mma(p2, dl[e], h0, h1);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) st[i][e] += p1[e] + p2[e];
        }
        publish_state();                                     // its readers of this chunk are behind the barrier above
        if (is_o) {
            float p[3][4];
#pragma unroll
            for (int i = 0; i < 3; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) p[i][e] = 0.f;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const uint32_t h0 = nt ? uh[1][2 * e] : uh[0][2 * e], h1 = nt ? uh[1][2 * e + 1] : uh[0][2 * e + 1];
                const uint32_t l0 = nt ? ul[1][2 * e] : ul[0][2 * e], l1 = nt ? ul[1][2 * e + 1] : ul[0][2 * e + 1];
                mma(p[0], ah[e], h0, h1);
                mma(p[1], ah[e], l0, l1);
                mma(p[2], al[e], h0, h1);
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = ch * C + mt * 16 + fr + 8 * e;
                if (t < n)
                    *(float2 *) (a.o + ((size_t) (r0 + t) * H + h) * V + vs * VB + nt * 8 + fc) =
                        make_float2(o[2 * e] + p[0][2 * e] + (p[1][2 * e] + p[2][2 * e]), o[2 * e + 1] + p[0][2 * e + 1] + (p[1][2 * e + 1] + p[2][2 * e + 1]));
            }
        }
        if (ch + 1 < chunks) load_rows(ch + 1);
        __syncthreads();                                     // S; this chunk's record is free
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (slot >= 0) {
#pragma unroll
        for (int i = 0; i < TPW; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) *(float2 *) (state + (size_t) (8 * e) * V + (sn0 + i) * 8) = make_float2(st[i][2 * e], st[i][2 * e + 1]);
    }
}

// SSD: 32 value columns per CTA; every warp owns a 16 x 8 tile of o and K / 32 tiles of S.  q and k are bf16, so only A, u and S are split.
constexpr int SV = 32, SB = SV + 8;                          // 80-byte rows hit different banks
template <int K> struct PassSsd {
    using R = Rec<SSD, K>;
    static constexpr int X = R::BYTES;                       // x bf16 [C][SV], factors fp32 [C]
    static constexpr int STAGE = X + C * SV * 2 + C * 4;
    static constexpr int S = STAGES * STAGE;                 // S hi, lo [K][SB]
    static constexpr int U = S + 2 * K * SB * 2;             // s x and its decayed form: hi, lo, hi, lo [C][SB]
    static constexpr int A = U + 4 * C * SB * 2;             // A hi, lo
    static constexpr int SMEM = A + 2 * R::ATILE;
};

template <int K>
__global__ void __launch_bounds__(NT, 1) chunk_pass_ssd_kernel(const __grid_constant__ jib_state_mix a) {
    using R = Rec<SSD, K>;
    using P = PassSsd<K>;
    constexpr int TPW = K / 32;
    extern __shared__ __align__(16) uint8_t smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int V = a.V, H = a.H, splits = (V + SV - 1) / SV, h = blockIdx.x / splits, v0 = blockIdx.x % splits * SV, b = blockIdx.y;
    const int units = min(SV, V - v0) / 8;                   // 8-column units that exist
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int r0 = a.q_start[b], n = a.q_start[b + 1] - r0;
    if (n <= 0) return;
    const int slot = checked_slot(a, b, 46), groups = H / a.rep;
    const int chunks = (n + C - 1) / C;
    const uint8_t * rec0 = (const uint8_t *) a.chunk + ((size_t) chunk_key(a.q_start, b) * groups + h / a.rep) * R::BYTES;
    auto stage = [&](int i) {
        if (i < chunks) {
            uint8_t * dst = smem + i % STAGES * P::STAGE;
            const uint8_t * src = rec0 + (size_t) i * groups * R::BYTES;
            for (int o = tid * 16; o < R::BYTES; o += NT * 16) cp16(dst + o, src + o);
            const int m = min(C, n - i * C), row = tid >> 2, u = tid & 3;
            if (row < m && u < units) cp16(dst + P::X + tid * 16, (const bf16 *) a.v + (size_t) (r0 + i * C + row) * H * V + h * V + v0 + u * 8);
            if (tid < m) cp4(dst + P::X + C * SV * 2 + tid * 4, a.s + (size_t) (r0 + i * C + tid) * H + h);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    stage(0);
    stage(1);
    store_conv_tail<bf16>(a, slot, r0, n, blockIdx.x * NT + tid, gridDim.x * NT);

    bf16 * Sh = (bf16 *) (smem + P::S), * Uh = (bf16 *) (smem + P::U);
    const uint32_t S_addr = sm100::smem_u32(Sh), U_addr = sm100::smem_u32(Uh), A_addr = sm100::smem_u32(smem + P::A);
    constexpr uint32_t S_LO = K * SB * 2, U_LO = C * SB * 2;
    const int fr = lane >> 2, fc = (lane & 3) * 2, lr = lane & 15, lu = lane >> 4;
    const int tr = (lane & 7) + ((lane >> 4) << 3), tu = (lane >> 3) & 1;
    const int mt = warp >> 2, nt = warp & 3;
    const int sm_ = warp * TPW >> 2, sn0 = TPW == 4 ? 0 : (warp & 1) * 2;
    float st[TPW][4];
    float * state = a.state + (((size_t) (slot < 0 ? 0 : slot) * H + h) * K + sm_ * 16 + fr) * V + v0 + fc;
    const bool past = slot >= 0 && a.positions[r0] > 0;
#pragma unroll
    for (int i = 0; i < TPW; ++i)
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const float2 x = past && sn0 + i < units ? *(const float2 *) (state + (size_t) (8 * e) * V + (sn0 + i) * 8) : make_float2(0.f, 0.f);
            st[i][2 * e] = x.x;
            st[i][2 * e + 1] = x.y;
        }
    auto publish_state = [&]() {
#pragma unroll
        for (int i = 0; i < TPW; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                uint32_t hi, lo;
                split2(st[i][2 * e], st[i][2 * e + 1], hi, lo);
                bf16 * p = Sh + (sm_ * 16 + fr + 8 * e) * SB + (sn0 + i) * 8 + fc;
                *(uint32_t *) p = hi;
                *(uint32_t *) (p + K * SB) = lo;
            }
    };
    uint32_t xq[K / 16][4], xk[2][4];                        // rows of q of this warp's tile; k^T of its tiles of S
    auto load_rows = [&](int ch) {
        const uint32_t rec = sm100::smem_u32(smem + ch % STAGES * P::STAGE);
        const int r = mt * 16 + lr;
#pragma unroll
        for (int kk = 0; kk < K / 16; ++kk) ldm4(xq[kk], rec + R::Q + r * (K * 2) + (((kk * 2 + lu) ^ (r & 7)) << 4));
    };
    const float na = a.neg_a[h] * LOG2E, skip = a.skip[h];
    publish_state();
    asm volatile("cp.async.wait_group 1;" ::: "memory");
    __syncthreads();
    load_rows(0);
    for (int ch = 0; ch < chunks; ++ch) {
        stage(ch + 2);                                       // into the buffer of chunk ch - 1
        const uint8_t * rec = smem + ch % STAGES * P::STAGE;
        const uint32_t rec_addr = sm100::smem_u32(rec);
        const int m = min(C, n - ch * C);
        const float * factor = (const float *) (rec + P::X + C * SV * 2);
        float acc[4][4];
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[i][e] = 0.f;
#pragma unroll
        for (int kk = 0; kk < K / 32; ++kk) {
            uint32_t bh[4], bl[4];
            const uint32_t off = ((kk * 32 + lane) * SB + nt * 8) * 2;
            ldm4t(bh, S_addr + off);
            ldm4t(bl, S_addr + S_LO + off);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                mma(acc[e], xq[2 * kk + e], bh[2 * e], bh[2 * e + 1]);
                mma(acc[2 + e], xq[2 * kk + e], bl[2 * e], bl[2 * e + 1]);
            }
        }
        // lane t: G_t
        float g = lane < m ? na * factor[lane] : 0.f;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float x = __shfl_up_sync(0xffffffffu, g, o);
            if (lane >= o) g += x;
        }
        const float gC = __shfl_sync(0xffffffffu, g, 31);
        {   // s x and s x e^{G_C - G}: 4 columns of a row per thread
            const int row = tid >> 3, c = (tid & 7) * 4;
            const float f = row < m ? factor[row] : 0.f, w = f * ex2(gC - __shfl_sync(0xffffffffu, g, row));
            float x[4] = {0.f, 0.f, 0.f, 0.f};
            if (row < m) load4((const bf16 *) (rec + P::X) + row * SV + c, x);
            uint2 hi, lo;
            bf16 * p = Uh + row * SB + c;
            split2(x[0] * f, x[1] * f, hi.x, lo.x);
            split2(x[2] * f, x[3] * f, hi.y, lo.y);
            *(uint2 *) p = hi;
            *(uint2 *) (p + C * SB) = lo;
            split2(x[0] * w, x[1] * w, hi.x, lo.x);
            split2(x[2] * w, x[3] * w, hi.y, lo.y);
            *(uint2 *) (p + 2 * C * SB) = hi;
            *(uint2 *) (p + 3 * C * SB) = lo;
        }
#pragma unroll
        for (int k = 0; k < C / 8; ++k) {                    // A = q . k times the decay between the two tokens: 4 rows per warp
            const int t = warp * (C / 8) + k;
            const float gt = __shfl_sync(0xffffffffu, g, t);                         // by all lanes, outside the condition
            const float x = lane <= t ? ((const float *) (rec + R::A))[t * QK_LD + lane] * ex2(gt - g) : 0.f;
            const bf16 hi = __float2bfloat16(x);
            *(bf16 *) (smem + P::A + a_off(t, lane)) = hi;
            *(bf16 *) (smem + P::A + R::ATILE + a_off(t, lane)) = __float2bfloat16(x - to_f(hi));
        }
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int r = e * 16 + tr;
            ldm4t(xk[e], rec_addr + R::D + r * (K * 2) + (((sm_ * 2 + tu) ^ (r & 7)) << 4));
        }
        asm volatile("cp.async.wait_group 1;" ::: "memory");
        __syncthreads();                                     // u, A, and the next chunk's record
        const float decay = ex2(gC);
#pragma unroll
        for (int i = 0; i < TPW; ++i) {
            uint32_t bh[4], bl[4];
            const uint32_t off = (lane * SB + (sn0 + i) * 8) * 2;
            ldm4t(bh, U_addr + 2 * U_LO + off);
            ldm4t(bl, U_addr + 3 * U_LO + off);
            float p1[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int e = 0; e < 4; ++e) st[i][e] *= decay;
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                mma(st[i], xk[e], bh[2 * e], bh[2 * e + 1]);
                mma(p1, xk[e], bl[2 * e], bl[2 * e + 1]);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) st[i][e] += p1[e];
        }
        publish_state();                                     // its readers of this chunk are behind the barrier above
        {
            float p[3][4];
#pragma unroll
            for (int i = 0; i < 3; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) p[i][e] = 0.f;
            uint32_t bh[4], bl[4], xh[4], xl[4];
            const float w0 = ex2(__shfl_sync(0xffffffffu, g, mt * 16 + fr)), w1 = ex2(__shfl_sync(0xffffffffu, g, mt * 16 + fr + 8));
            const uint32_t off = (lane * SB + nt * 8) * 2;
            ldm4t(bh, U_addr + off);
            ldm4t(bl, U_addr + U_LO + off);
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int r = mt * 16 + lr;
                const uint32_t q = A_addr + r * 64 + (((e * 2 + lu) ^ ((r >> 1) & 3)) << 4);
                ldm4(xh, q);
                ldm4(xl, q + R::ATILE);
                mma(p[0], xh, bh[2 * e], bh[2 * e + 1]);
                mma(p[1], xh, bl[2 * e], bl[2 * e + 1]);
                mma(p[2], xl, bh[2 * e], bh[2 * e + 1]);
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
                const int t = mt * 16 + fr + 8 * e, c = nt * 8 + fc;
                const float w = e ? w1 : w0;
                if (t >= m || nt >= units) continue;
                const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *) (rec + P::X + (t * SV + c) * 2));
                float2 y;
                y.x = w * ((acc[0][2 * e] + acc[1][2 * e]) + (acc[2][2 * e] + acc[3][2 * e])) + p[0][2 * e] + (p[1][2 * e] + p[2][2 * e]) + skip * x.x;
                y.y = w * ((acc[0][2 * e + 1] + acc[1][2 * e + 1]) + (acc[2][2 * e + 1] + acc[3][2 * e + 1])) + p[0][2 * e + 1] +
                      (p[1][2 * e + 1] + p[2][2 * e + 1]) + skip * x.y;
                *(float2 *) (a.o + ((size_t) (r0 + ch * C + t) * H + h) * V + v0 + c) = y;
            }
        }
        if (ch + 1 < chunks) load_rows(ch + 1);
        __syncthreads();                                     // S; this chunk's record is free
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (slot >= 0) {
#pragma unroll
        for (int i = 0; i < TPW; ++i)
#pragma unroll
            for (int e = 0; e < 2; ++e)
                if (sn0 + i < units) *(float2 *) (state + (size_t) (8 * e) * V + (sn0 + i) * 8) = make_float2(st[i][2 * e], st[i][2 * e + 1]);
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

// The passes are plain launches: as programmatic dependents their CTAs would settle wherever the last CTAs of prepare leave room,
// several to an SM.
template <int KIND, int K> int run_chunks(const jib_state_mix & a, cudaStream_t s) {
    const int nch = a.T / C + a.n_seqs;
    static std::atomic<unsigned char> done1[jib::MAX_DEVICES], done2[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(chunk_prepare_kernel<KIND, K>, prep_smem<K>(256), done1)) return JIB_E_LAUNCH;
    JIB_LAUNCH((chunk_prepare_kernel<KIND, K>), dim3(nch, a.H), NT, prep_smem<K>(a.V), s, a);
    const int rc = launched();
    if (rc) return rc;
    if (!jib::ensure_dyn_smem(chunk_pass_kernel<KIND, K>, Pass<KIND, K>::SMEM, done2)) return JIB_E_LAUNCH;
    chunk_pass_kernel<KIND, K><<<dim3(a.H * (a.V / VB), a.n_seqs), NT, Pass<KIND, K>::SMEM, s>>>(a);
    return launched();
}
template <int K> int run_chunks_ssd(const jib_state_mix & a, cudaStream_t s) {
    const int nch = a.T / C + a.n_seqs;
    static std::atomic<unsigned char> done1[jib::MAX_DEVICES], done2[jib::MAX_DEVICES];
    constexpr int smem = 2 * C * (K + 4) * 4;
    if (!jib::ensure_dyn_smem(chunk_prepare_ssd_kernel<K>, smem, done1)) return JIB_E_LAUNCH;
    JIB_LAUNCH((chunk_prepare_ssd_kernel<K>), dim3(nch, a.H / a.rep + (a.H * a.V + 255) / 256 + 1), NT, smem, s, a);
    const int rc = launched();
    if (rc) return rc;
    if (!jib::ensure_dyn_smem(chunk_pass_ssd_kernel<K>, PassSsd<K>::SMEM, done2)) return JIB_E_LAUNCH;
    chunk_pass_ssd_kernel<K><<<dim3(a.H * ((a.V + SV - 1) / SV), a.n_seqs), NT, PassSsd<K>::SMEM, s>>>(a);
    return launched();
}

long long rec_bytes(const jib_state_mix & a) {
#define REC(KIND) (a.K == 64 ? Rec<KIND, 64>::BYTES : Rec<KIND, 128>::BYTES)
    const long long nch = a.T / C + a.n_seqs;
    if (a.kind == SSD) return nch * (a.H / a.rep) * REC(SSD);
    return nch * a.H * ((a.kind == DELTA ? REC(DELTA) : REC(LINEAR)) + C * 4 * a.V);
#undef REC
}

}  // namespace

bool jib_state_chunk_ok(const jib_state_mix & a) {
    const long long cols = a.ld | a.q_off | a.k_off | a.v_off | a.conv0 | a.n_conv | (a.kind == SSD ? 0 : a.ld_dec);
    return (a.K == 64 || a.K == 128) && a.V % VB == 0 && a.V <= 256 && a.taps <= 4 && cols % 4 == 0 && ((uintptr_t) a.proj & 7) == 0 &&
           (a.kind == SSD || ((uintptr_t) a.dec_in & 7) == 0) && a.H % a.rep == 0;
}

int jib_state_chunk_run(const jib_state_mix & a, cudaStream_t s) {
    if (rec_bytes(a) > a.chunk_bytes) return JIB_E_SCRATCH;
    switch (a.kind) {
        case DELTA: return a.K == 64 ? run_chunks<DELTA, 64>(a, s) : run_chunks<DELTA, 128>(a, s);
        case LINEAR: return a.K == 64 ? run_chunks<LINEAR, 64>(a, s) : run_chunks<LINEAR, 128>(a, s);
        default: return a.K == 64 ? run_chunks_ssd<64>(a, s) : run_chunks_ssd<128>(a, s);
    }
}

// Bytes of scratch (m->chunk) with which jib_state_mix_run takes a batch of portions through the tensor cores; 0: not these sizes.
extern "C" JIB_EXPORT long long jib_state_chunk_bytes(const jib_state_mix * m) { return jib_state_chunk_ok(*m) ? rec_bytes(*m) : 0; }
