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
//   HGRN is LINEAR with q, k and decays of its own; MLSTM is SSD without groups whose decays and factors mlstm_gates has written, with one more
//   value column (v = 1): the state of that column is what the keys add up to.
//   pass    (K / 32 warps per head and 16 value columns): walks the chunks, S in registers, everything else a product of small matrices.
// State, decays, A, W, U0 are fp32; the tensor cores see each as a sum of two bf16 numbers and the products hi * hi + hi * lo + lo * hi
// (about 16 bits of mantissa); q and k of SSD are bf16 to begin with.  Accumulation is fp32.
#include "pdl.cuh"
#include "state_mix.cuh"

namespace {

using namespace state_mix;

constexpr int C = 32, NT = 256;                              // tokens of a chunk; threads of prepare
constexpr float LOG2E = 1.4426950408889634f;
__host__ __device__ constexpr bool per_head(int kind) { return !per_channel(kind); }       // SSD, MLSTM

// A chunk's record: bf16 tiles of 32 rows x K columns in 16-byte units u of row r stored at u ^ (r & 7); A: 32 x 32, unit u ^ (r / 2 & 3).
template <int KIND, int K> struct Rec {
    static constexpr int TILE = C * K * 2, ATILE = C * C * 2;
    static constexpr int Q = 0, D = per_head(KIND) ? TILE : 2 * TILE;                     // q e^G, k e^{G_C - G} (SSD: q, k)
    static constexpr int A = per_head(KIND) ? 2 * TILE : 4 * TILE;                        // hi, lo
    static constexpr int W = A + 2 * ATILE;                                               // DELTA
    static constexpr int E = W + (KIND == DELTA ? 2 * TILE : 0);                          // e^{G_C}; SSD: e^{G_t}, then s_t e^{G_C - G_t}
    static constexpr int BYTES = E + (per_head(KIND) ? 2 * C : K) * 4;
};
// SSD: q and k (the first A bytes) are shared by a group; the rest is per head and lies behind all groups' parts.
template <int K> __device__ __forceinline__ uint8_t * ssd_group_part(const jib_state_mix & a, int ci, int group) {
    return (uint8_t *) a.chunk + ((size_t) ci * (a.H / a.rep) + group) * Rec<SSD, K>::A;
}
template <int K> __device__ __forceinline__ uint8_t * ssd_head_part(const jib_state_mix & a, int ci, int h) {
    using R = Rec<SSD, K>;
    return (uint8_t *) a.chunk + (size_t) (a.T / C + a.n_seqs) * (a.H / a.rep) * R::A + ((size_t) ci * a.H + h) * (R::BYTES - R::A);
}

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
        if (KIND == HGRN && j >= jk && j < 2 * jk + jv) continue;              // k comes with the decays, the pass reads the values where they are
        if (j < 2 * jk + jv) {
            const int jj = j < jk ? j : j < 2 * jk ? j - jk : j - 2 * jk, w = j < 2 * jk ? K / 4 : V / 4;
            col = jj % w * 4;
            run = jj / w * 8;
            ld = j < 2 * jk ? KS : VS;
            dst = j < jk ? q : j < 2 * jk ? k : v;
            conv_run(a, r0, p0, nr, t0 + run, (j < jk ? a.q_off + h / a.rep * K : j < 2 * jk ? a.k_off + h / a.rep * K : a.v_off + h * V) + col, slot, x);
            if (KIND == HGRN) {
#pragma unroll
                for (int r = 0; r < 8; ++r)
#pragma unroll
                    for (int e = 0; e < 4; ++e) x[r][e] = silu<bf16>(x[r][e]);
            }
            if (KIND == LINEAR && j >= 2 * jk) {             // values as they are
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    if (run + r >= n) break;
                    __nv_bfloat162 y[2] = {__floats2bfloat162_rn(x[r][0], x[r][1]), __floats2bfloat162_rn(x[r][2], x[r][3])};
                    *(uint2 *) ((bf16 *) a.v + ((size_t) (r0 + t0 + run + r) * a.H + h) * V + col) = *(const uint2 *) y;
                }
                continue;
            }
        } else {
            const int jj = j - 2 * jk - jv;
            col = jj % (K / 4) * 4;
            run = jj / (K / 4) * 8;
            ld = KS;
            dst = G;
            const bf16 * z = (const bf16 *) a.dec_in + (size_t) (r0 + t0) * a.ld_dec + h * K + col;
            const float4 bias = *(const float4 *) (a.bias + h * K + col);
            const float f = KIND == HGRN ? 0.f : LOG2E * (KIND == DELTA ? a.neg_a[h] : -a.inv_tau);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
#pragma unroll
                for (int e = 0; e < 4; ++e) x[r][e] = 0.f;
                if (run + r < n) load4(z + (size_t) (run + r) * a.ld_dec, x[r]);
            }
            if (KIND == HGRN) {
                const float4 l4 = *(const float4 *) (a.lower + h * K + col);
                const float l[4] = {l4.x, l4.y, l4.z, l4.w}, bz[4] = {bias.x, bias.y, bias.z, bias.w};
#pragma unroll
                for (int r = 0; r < 8; ++r) {
                    float y[4];
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        float g, rest;
                        bounded_gate(x[r][e] + bz[e], l[e], g, rest);
                        const bool in = run + r < n;
                        y[e] = in ? rest : 0.f;              // log f to a few ulp: near 1 from 1 - f
                        x[r][e] = in ? LOG2E * (rest < 0.5f ? log1pf(-rest) : logf(fmaxf(g, 1e-37f))) : 0.f;
                    }
                    *(float4 *) (k + (run + r) * KS + col) = make_float4(y[0], y[1], y[2], y[3]);
                }
            }
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                if (KIND == HGRN) break;
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
        float ss[2 * C / (NT / 32)];                         // 8 rows per warp, their reductions side by side
#pragma unroll
        for (int i = 0; i < 2 * C / (NT / 32); ++i) {
            const int r = warp + i * (NT / 32);
            const float * x = (r < C ? q : k) + (r & (C - 1)) * KS;
            ss[i] = 0.f;
#pragma unroll
            for (int c = lane; c < K; c += 32) ss[i] += x[c] * x[c];
        }
#pragma unroll
        for (int i = 0; i < 2 * C / (NT / 32); ++i) ss[i] = warp_sum(ss[i]);
        if (lane == 0)
#pragma unroll
            for (int i = 0; i < 2 * C / (NT / 32); ++i) {
                const int r = warp + i * (NT / 32);
                norm[r] = rsqrtf(ss[i] + 1e-6f) * (r < C ? a.q_scale : 1.f);
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
    uint8_t * rec = (uint8_t *) a.chunk + ((size_t) ci * a.H + h) * (R::BYTES + (KIND == DELTA ? C * 4 * V : 0));
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
    float dg[C / (NT / 32)];                                 // the diagonal
#pragma unroll
    for (int i = 0; i < C / (NT / 32); ++i) {
        const int t = warp + i * (NT / 32);
        dg[i] = 0.f;
#pragma unroll
        for (int c = lane; c < K; c += 32) dg[i] += q[t * KS + c] * k[t * KS + c];
    }
#pragma unroll
    for (int i = 0; i < C / (NT / 32); ++i) {
        const int t = warp + i * (NT / 32);
        const float d = warp_sum(dg[i]);
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
    if (KIND != DELTA) return;
    float * U = (float *) (rec + R::BYTES);
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
            for (int t = 0; t < C; ++t) U[(cc >> 4) * (C * 16) + t * 16 + (cc & 15)] = x[t];
        }
    }
}

// ---- prepare: SSD ------------------------------------------------------------------------------------------------------------------
// blockIdx.y < groups * blocks of 16 heads: q and k tiles of a group and their products, then A and the decays of 16 heads of the group
// (A_ts also holds the factor s_s of the earlier token, and D on the diagonal).  Then runs of 256 value columns (bf16 into a.v).
constexpr int HB = 16;

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
    const int blocks = (a.rep + HB - 1) / HB;
    int y = blockIdx.y;
    if (y < groups * blocks) {
        float * q = sm, * k = sm + C * KS, * qk = k + C * KS;             // qk [C][C + 1]
        const int block = y % blocks;
        y /= blocks;
        uint8_t * rec = ssd_group_part<K>(a, ci, y);
        const int jk = K / 4 * (C / 8);
        for (int j = tid; j < 2 * jk; j += NT) {
            float x[8][4];
            const int jj = j < jk ? j : j - jk, col = jj % (K / 4) * 4, run = jj / (K / 4) * 8;
            conv_run(a, r0, p0, nr, t0 + run, (j < jk ? a.q_off : a.k_off) + y * K + col, slot, x);
#pragma unroll
            for (int r = 0; r < 8; ++r) {
                __nv_bfloat162 v[2] = {__floats2bfloat162_rn(x[r][0], x[r][1]), __floats2bfloat162_rn(x[r][2], x[r][3])};
                if (block == 0) *(uint2 *) (rec + (j < jk ? R::Q : R::D) + tile_off<K>(run + r, col)) = *(const uint2 *) v;
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
            qk[t * (C + 1) + s] = d;
        }
        __syncthreads();
        const int lane = tid & 31;
        for (int i = tid >> 5; i < HB && block * HB + i < a.rep; i += NT / 32) {
            const int h = y * a.rep + block * HB + i;
            uint8_t * hr = ssd_head_part<K>(a, ci, h);
            const float f = lane < n ? softplus_series(to_f(((const bf16 *) a.proj)[(size_t) (r0 + t0 + lane) * a.ld + a.s_off + h]) + a.bias[h]) : 0.f;
            float g = a.neg_a[h] * LOG2E * f;                // lane t: G_t
#pragma unroll
            for (int o = 1; o < 32; o <<= 1) {
                const float x = __shfl_up_sync(0xffffffffu, g, o);
                if (lane >= o) g += x;
            }
            const float gC = __shfl_sync(0xffffffffu, g, 31), skip = a.skip[h];
            float * e = (float *) (hr + R::E - R::A);
            e[lane] = ex2(g);
            e[C + lane] = f * ex2(gC - g);
#pragma unroll 4
            for (int t = 0; t < C; ++t) {
                const float gt = __shfl_sync(0xffffffffu, g, t);
                float x = lane <= t ? qk[t * (C + 1) + lane] * (ex2(gt - g) * f) : 0.f;
                if (lane == t) x += skip;
                const bf16 hi = __float2bfloat16(x);
                *(bf16 *) (hr + a_off(t, lane)) = hi;
                *(bf16 *) (hr + R::ATILE + a_off(t, lane)) = __float2bfloat16(x - to_f(hi));
            }
        }
        return;
    }
    y -= groups * blocks;
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
}

// ---- prepare: MLSTM ----------------------------------------------------------------------------------------------------------------
// One CTA per chunk and head: q and k as they are, their products on the tensor cores (a warp per 16 x 8 of them), times decays and factors.
template <int K>
__global__ void __launch_bounds__(NT) chunk_prepare_mlstm_kernel(const __grid_constant__ jib_state_mix a) {
    using R = Rec<MLSTM, K>;
    __shared__ __align__(16) uint8_t tiles[2 * R::TILE];
    PDL_TRIGGER_TOP();
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int ci = blockIdx.x, h = blockIdx.y, b = chunk_seq(a, ci);
    const int r0 = a.q_start[b], nr = a.q_start[b + 1] - r0, t0 = (ci - chunk_key(a.q_start, b)) * C;
    if (t0 < 0 || t0 >= nr) return;
    const int n = min(C, nr - t0);
    uint8_t * rec = ssd_group_part<K>(a, ci, h), * hr = ssd_head_part<K>(a, ci, h);
    const bf16 * x = (const bf16 *) a.proj + (size_t) (r0 + t0) * a.ld + h * K;
    constexpr int U = K / 8;                                 // 16-byte units of a row
    uint4 v[2 * C * U / NT];
#pragma unroll
    for (int i = 0; i < 2 * C * U / NT; ++i) {
        const int j = tid + i * NT, r = j / U % C, u = j % U;
        v[i] = make_uint4(0, 0, 0, 0);
        if (r < n) v[i] = *(const uint4 *) (x + (size_t) r * a.ld + (j < C * U ? a.q_off : a.k_off) + u * 8);
    }
    float f = 0.f, g = 0.f;                                  // lane t: s_t, G_t
    if (lane < n) {
        const size_t at = (size_t) (r0 + t0 + lane) * a.H + h;
        f = a.s[at];
        g = a.dec[at];
    }
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const float y = __shfl_up_sync(0xffffffffu, g, o);
        if (lane >= o) g += y;
    }
    const float gC = __shfl_sync(0xffffffffu, g, 31);
    if (warp == 0) {
        float * e = (float *) (hr + R::E - R::A);
        e[lane] = ex2(g);
        e[C + lane] = f * ex2(gC - g);
    }
#pragma unroll
    for (int i = 0; i < 2 * C * U / NT; ++i) {
        const int j = tid + i * NT, r = j / U % C, u = j % U, off = (j < C * U ? R::Q : R::D) + tile_off<K>(r, u * 8);
        *(uint4 *) (tiles + off) = v[i];
        *(uint4 *) (rec + off) = v[i];
    }
    __syncthreads();
    const int mt = warp >> 2, nt = warp & 3;                 // rows (later tokens) 16 mt .., columns (earlier ones) 8 nt ..
    const uint32_t base = sm100::smem_u32(tiles);
    float c[4] = {0.f, 0.f, 0.f, 0.f};
    if (8 * nt <= 16 * mt + 15) {
#pragma unroll
        for (int kk = 0; kk < K; kk += 32) {
            uint32_t p[4], q[4], y[4];
            const int r = mt * 16 + (lane & 15), s = nt * 8 + (lane & 7);
            ldm4(p, base + R::Q + tile_off<K>(r, kk + (lane >> 4) * 8));
            ldm4(q, base + R::Q + tile_off<K>(r, kk + 16 + (lane >> 4) * 8));
            ldm4(y, base + R::D + tile_off<K>(s, kk + (lane >> 3) * 8));
            mma(c, p, y[0], y[1]);
            mma(c, q, y[2], y[3]);
        }
    }
    const int s0 = nt * 8 + (lane & 3) * 2;
    const float g0 = __shfl_sync(0xffffffffu, g, s0), g1 = __shfl_sync(0xffffffffu, g, s0 + 1);
    const float f0 = __shfl_sync(0xffffffffu, f, s0), f1 = __shfl_sync(0xffffffffu, f, s0 + 1);
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = mt * 16 + (lane >> 2) + 8 * e;
        const float gt = __shfl_sync(0xffffffffu, g, t);
        uint32_t hi, lo;
        split2(s0 <= t ? c[2 * e] * (ex2(gt - g0) * f0) : 0.f, s0 + 1 <= t ? c[2 * e + 1] * (ex2(gt - g1) * f1) : 0.f, hi, lo);
        *(uint32_t *) (hr + a_off(t, s0)) = hi;
        *(uint32_t *) (hr + R::ATILE + a_off(t, s0)) = lo;
    }
}

// ---- pass --------------------------------------------------------------------------------------------------------------------------
template <int KIND, int K> struct Pass {
    using R = Rec<KIND, K>;
    static constexpr int KS = K / 32;                        // warps that share a head's 16 value columns, 32 key channels each
    static constexpr int NG = (KIND == SSD ? 8 : 4) / KS;    // groups of 16 columns
    static constexpr int WARPS = KS * NG, PT = WARPS * 32, PV = NG * 16;
    static constexpr int STAGES = KIND == DELTA ? 3 : 4;
    static constexpr int XS = PV * 2 + 16;                   // bytes of a row of v: rows hit different banks
    static constexpr int X = R::BYTES;                       // v bf16 [C][PV] in rows of XS; DELTA: U0 fp32 [NG][C][16]
    static constexpr int STAGE = X + (KIND == DELTA ? NG * C * 16 * 4 : C * XS);
    static constexpr int O = STAGES * STAGE;                 // partial o^T [WARPS][4][32] float4, then (DELTA) of W S
    static constexpr int SMEM = O + WARPS * 2048 * (KIND == DELTA ? 2 : 1);
};

// 16 value columns of a head belong to K / 32 warps; each keeps its channels of S^T (16 x 32) in registers as the accumulators of
// S^T += u^T k.  In the products o^T = S^T q^T and S^T W^T those accumulators are the left operand as they stand (two m16n8 results are
// an m16k16 operand), and u^T, the result of one product, is the left operand of the next two.  Only the partial sums over the channels
// pass through shared memory.  Two barriers per chunk: the record is there; the partial sums are there.
template <int KIND, int K>
__global__ void __launch_bounds__(Pass<KIND, K>::PT, 1) chunk_pass_kernel(const __grid_constant__ jib_state_mix a) {
    using R = Rec<KIND, K>;
    using P = Pass<KIND, K>;
    constexpr int ST = P::STAGES, KS = P::KS, PT = P::PT, PV = P::PV;
    constexpr bool HEAD = per_head(KIND);
    extern __shared__ __align__(16) uint8_t smem[];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, V = a.V, H = a.H, VS = scratch_cols(KIND, V);
    const int NC = V + (KIND == MLSTM ? 16 : 0);             // value columns, those of the keys' sum last
    // values: rows of proj, or (after a convolution) of a.v
    const bf16 * val = KIND == HGRN || KIND == MLSTM ? (const bf16 *) a.proj + a.v_off : (const bf16 *) a.v;
    const size_t ldv = KIND == HGRN || KIND == MLSTM ? (size_t) a.ld : (size_t) H * V;
    const int splits = (NC + PV - 1) / PV, h = blockIdx.x / splits, v0 = blockIdx.x % splits * PV, b = blockIdx.y;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int r0 = a.q_start[b], n = a.q_start[b + 1] - r0;
    if (n <= 0) return;
    const int slot = checked_slot(a, b, 46), chunks = (n + C - 1) / C;
    const int units = min(PV, NC - v0) / 8;                  // 8-column units that exist
    const int grp = warp / KS, ks = warp % KS;               // this warp's columns and channels
    const bool active = grp * 2 < units;
    const size_t rec_bytes = R::BYTES + (KIND == DELTA ? C * 4 * V : 0);
    const int c0 = chunk_key(a.q_start, b);
    auto stage = [&](int i) {
        if (i < chunks) {
            uint8_t * dst = smem + i % ST * P::STAGE;
            const uint8_t * src = HEAD ? ssd_group_part<K>(a, c0 + i, h / a.rep) : (const uint8_t *) a.chunk + ((size_t) (c0 + i) * H + h) * rec_bytes;
#pragma unroll 4
            for (int o = tid * 16; o < (HEAD ? R::A : R::BYTES); o += PT * 16) cp16(dst + o, src + o);
            if (HEAD) {
                const uint8_t * hr = ssd_head_part<K>(a, c0 + i, h);
                for (int o = tid * 16; o < R::BYTES - R::A; o += PT * 16) cp16(dst + R::A + o, hr + o);
            }
            if (KIND == DELTA) {
                for (int o = tid * 16; o < units / 2 * (C * 64); o += PT * 16) cp16(dst + P::X + o, src + R::BYTES + v0 / 16 * (C * 64) + o);
            } else {
                const int m = min(C, n - i * C);
                for (int j = tid; j < C * (PV / 8); j += PT) {
                    const int row = j / (PV / 8), u = j % (PV / 8);
                    if (row >= m) *(uint4 *) (dst + P::X + row * P::XS + (u << 4)) = make_uint4(0, 0, 0, 0);
                    else if (KIND == MLSTM && v0 + u * 8 >= V)                 // 1, then zeros
                        *(uint4 *) (dst + P::X + row * P::XS + (u << 4)) = make_uint4(v0 + u * 8 == V ? 0x3f80 : 0, 0, 0, 0);
                    else if (u < units)
                        cp16(dst + P::X + row * P::XS + (u << 4), val + (size_t) (r0 + i * C + row) * ldv + h * V + v0 + u * 8);
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
#pragma unroll
    for (int i = 0; i < ST - 1; ++i) stage(i);
    store_conv_tail<bf16>(a, slot, r0, n, blockIdx.x * PT + tid, gridDim.x * PT);

    const int fr = lane >> 2, fc = (lane & 3) * 2;           // accumulator element: rows fr, fr + 8 (values), columns fc, fc + 1
    const int tr = (lane & 7) + ((lane >> 4) << 3), tu = (lane >> 3) & 1;
    float st[4][4];                                          // 4 tiles of 8 channels
    const bool sum = KIND == MLSTM && v0 + grp * 16 >= V;    // the columns of the keys' sum, of which one exists
    const size_t row_at = ((size_t) (slot < 0 ? 0 : slot) * H + h), lds = sum ? 1 : V;
    float * state = sum ? a.extra + row_at * (K + 1) + ks * 32 : a.state + (row_at * K + ks * 32) * V + v0 + grp * 16 + fr;
    const bool past = slot >= 0 && a.positions[r0] > 0 && active;
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < 4; ++e) st[i][e] = past && (!sum || (fr == 0 && e < 2)) ? state[(i * 8 + fc + (e & 1)) * lds + 8 * (e >> 1)] : 0.f;
    for (int ch = 0; ch < chunks; ++ch) {
        asm volatile("cp.async.wait_group %0;" ::"n"(ST - 2) : "memory");
        __syncthreads();                                     // this chunk's record is there; the oldest is free
        stage(ch + ST - 1);
        const uint8_t * rec = smem + ch % ST * P::STAGE;
        const uint32_t rec_addr = sm100::smem_u32(rec);
        const uint32_t A_addr = rec_addr + R::A;
        float4 * part = (float4 *) (smem + P::O) + warp * 128 + lane;          // this warp's partial sums: [4 token tiles][32 lanes]
        uint32_t xh[2][4], xl[2][4], yh[2][4], yl[2][4];     // u^T, hi and lo, 16 tokens at a time (x: of the read-out, y: of the update)
        const float * eg = (const float *) (rec + R::E), * wt = eg + C;        // SSD, MLSTM
        const float dC = HEAD ? eg[C - 1] : 0.f;
        if (active) {
            float o[4][4], w[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i)
#pragma unroll
                for (int e = 0; e < 4; ++e) o[i][e] = w[i][e] = 0.f;
            uint32_t sh[2][4], sl[2][4];
#pragma unroll
            for (int j = 0; j < 2; ++j)
#pragma unroll
                for (int i = 0; i < 4; ++i) split2(st[2 * j + (i >> 1)][2 * (i & 1)], st[2 * j + (i >> 1)][2 * (i & 1) + 1], sh[j][i], sl[j][i]);
            uint32_t y[4][4], z[4][4];
            auto rows = [&](uint32_t (&t)[4][4], uint32_t tile) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const int r = i * 8 + (lane & 7);
                    ldm4(t[i], rec_addr + tile + r * (K * 2) + (((ks * 4 + (lane >> 3)) ^ (r & 7)) << 4));
                }
            };
            if (KIND == DELTA) rows(z, R::W);
            rows(y, R::Q);
            // in an order that keeps four (DELTA: eight) accumulators in flight
#pragma unroll
            for (int j = 0; j < 2; ++j) {
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (KIND == DELTA) mma(w[i], sh[j], z[i][2 * j], z[i][2 * j + 1]);
                    mma(o[i], sh[j], y[i][2 * j], y[i][2 * j + 1]);
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (KIND == DELTA) mma(w[i], sl[j], z[i][2 * j], z[i][2 * j + 1]);
                    mma(o[i], sl[j], y[i][2 * j], y[i][2 * j + 1]);
                }
            }
            if (!HEAD) {
                if (KIND == DELTA) rows(z, R::W + R::TILE);
                rows(y, R::Q + R::TILE);
#pragma unroll
                for (int j = 0; j < 2; ++j)
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (KIND == DELTA) mma(w[i], sh[j], z[i][2 * j], z[i][2 * j + 1]);
                        mma(o[i], sh[j], y[i][2 * j], y[i][2 * j + 1]);
                    }
            }
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                part[i * 32] = make_float4(o[i][0], o[i][1], o[i][2], o[i][3]);
                if (KIND == DELTA) part[P::WARPS * 128 + i * 32] = make_float4(w[i][0], w[i][1], w[i][2], w[i][3]);
            }
        }
        if (KIND == DELTA) __syncthreads();
        if (active) {
            if (KIND == DELTA) {                             // u^T = U0^T - S^T W^T
                const float4 * all = (const float4 *) (smem + P::O) + (P::WARPS + grp * KS) * 128 + lane;
                const float * u0 = (const float *) (rec + P::X) + grp * (C * 16) + fr;
                float u[4][4];
#pragma unroll
                for (int i = 0; i < 4; ++i) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) u[i][e] = u0[(i * 8 + fc + (e & 1)) * 16 + 8 * (e >> 1)];
#pragma unroll
                    for (int k = 0; k < KS; ++k) {
                        const float4 p = all[k * 128 + i * 32];
                        u[i][0] -= p.x; u[i][1] -= p.y; u[i][2] -= p.z; u[i][3] -= p.w;
                    }
                }
#pragma unroll
                for (int e = 0; e < 2; ++e)
#pragma unroll
                    for (int i = 0; i < 4; ++i) split2(u[2 * e + (i >> 1)][2 * (i & 1)], u[2 * e + (i >> 1)][2 * (i & 1) + 1], xh[e][i], xl[e][i]);
            } else {
#pragma unroll
                for (int e = 0; e < 2; ++e) ldm4t(xh[e], rec_addr + P::X + (e * 16 + tr) * P::XS + ((grp * 2 + tu) << 4));
            }
            if (HEAD) {
#pragma unroll
                for (int e = 0; e < 2; ++e)
#pragma unroll
                    for (int j = 0; j < 2; ++j) {            // tokens 16 e + 8 j + fc, + 1
                        const float2 wj = *(const float2 *) (wt + e * 16 + j * 8 + fc);
#pragma unroll
                        for (int i = 2 * j; i < 2 * j + 2; ++i) {
                            const float2 x = __bfloat1622float2(*(const __nv_bfloat162 *) &xh[e][i]);
                            split2(x.x * wj.x, x.y * wj.y, yh[e][i], yl[e][i]);
                        }
                    }
            }
            // S^T <- decay S^T + u^T k
            uint32_t y[4][4], z[4][4];
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const uint32_t off = lane * (K * 2) + (((ks * 4 + i) ^ (lane & 7)) << 4);
                ldm4t(y[i], rec_addr + R::D + off);
                if (!HEAD) ldm4t(z[i], rec_addr + R::D + R::TILE + off);
                float2 d = make_float2(dC, dC);
                if (!HEAD) d = *(const float2 *) (rec + R::E + (ks * 32 + i * 8 + fc) * 4);
                st[i][0] *= d.x; st[i][1] *= d.y; st[i][2] *= d.x; st[i][3] *= d.y;
            }
#pragma unroll
            for (int e = 0; e < 2; ++e) {
#pragma unroll
                for (int i = 0; i < 4; ++i) mma(st[i], HEAD ? yh[e] : xh[e], y[i][2 * e], y[i][2 * e + 1]);
                if (KIND == DELTA || HEAD) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) mma(st[i], HEAD ? yl[e] : xl[e], y[i][2 * e], y[i][2 * e + 1]);
                }
                if (!HEAD) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) mma(st[i], xh[e], z[i][2 * e], z[i][2 * e + 1]);
                }
            }
        }
        if (KIND != DELTA) __syncthreads();
        if (active) {                                        // o^T of 4 / KS token tiles: the partial sums, then += u^T A^T
#pragma unroll
            for (int k = 0; k < 4 / KS; ++k) {
                const int i = ks * (4 / KS) + k, r = i * 8 + (lane & 7);
                const float4 * all = (const float4 *) (smem + P::O) + grp * KS * 128 + i * 32 + lane;
                float o[4] = {0.f, 0.f, 0.f, 0.f}, q[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int p = 0; p < KS; ++p) {
                    const float4 x = all[p * 128];
                    o[0] += x.x; o[1] += x.y; o[2] += x.z; o[3] += x.w;
                }
                if (HEAD) {
                    const float2 e = *(const float2 *) (eg + i * 8 + fc);
                    o[0] *= e.x; o[1] *= e.y; o[2] *= e.x; o[3] *= e.y;
                }
                const uint32_t off = r * 64 + (((lane >> 3) ^ ((r >> 1) & 3)) << 4);
                uint32_t y[4], z[4];
                ldm4(y, A_addr + off);
                ldm4(z, A_addr + R::ATILE + off);
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    mma(o, xh[e], y[2 * e], y[2 * e + 1]);
                    mma(q, xh[e], z[2 * e], z[2 * e + 1]);
                    if (KIND == DELTA) mma(q, xl[e], y[2 * e], y[2 * e + 1]);
                }
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const int t = ch * C + i * 8 + fc + (e & 1);
                    if (t < n && (!sum || (fr == 0 && e < 2))) a.o[((size_t) (r0 + t) * H + h) * VS + v0 + grp * 16 + fr + 8 * (e >> 1)] = o[e] + q[e];
                }
            }
        }
    }
    asm volatile("cp.async.wait_group 0;" ::: "memory");
    if (slot >= 0 && active) {
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (!sum || (fr == 0 && e < 2)) state[(i * 8 + fc + (e & 1)) * lds + 8 * (e >> 1)] = st[i][e];
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

// The pass is a plain launch: as a programmatic dependent its CTAs would settle wherever the last CTAs of prepare leave room, several
// to an SM.
template <int KIND, int K> int launch_pass(const jib_state_mix & a, cudaStream_t s) {
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(chunk_pass_kernel<KIND, K>, Pass<KIND, K>::SMEM, done)) return JIB_E_LAUNCH;
    chunk_pass_kernel<KIND, K><<<dim3(a.H * ((a.V + (KIND == MLSTM ? 16 : 0) + Pass<KIND, K>::PV - 1) / Pass<KIND, K>::PV), a.n_seqs), Pass<KIND, K>::PT, Pass<KIND, K>::SMEM, s>>>(a);
    return launched();
}
template <int KIND, int K> int run_chunks(const jib_state_mix & a, cudaStream_t s) {
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(chunk_prepare_kernel<KIND, K>, prep_smem<K>(256), done)) return JIB_E_LAUNCH;
    JIB_LAUNCH((chunk_prepare_kernel<KIND, K>), dim3(a.T / C + a.n_seqs, a.H), NT, prep_smem<K>(a.V), s, a);
    const int rc = launched();
    return rc ? rc : launch_pass<KIND, K>(a, s);
}
template <int K> int run_chunks_mlstm(const jib_state_mix & a, cudaStream_t s) {
    JIB_LAUNCH((chunk_prepare_mlstm_kernel<K>), dim3(a.T / C + a.n_seqs, a.H), NT, 0, s, a);
    const int rc = launched();
    return rc ? rc : launch_pass<MLSTM, K>(a, s);
}
template <int K> int run_chunks_ssd(const jib_state_mix & a, cudaStream_t s) {
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    constexpr int smem = (2 * C * (K + 4) + C * (C + 1)) * 4;
    if (!jib::ensure_dyn_smem(chunk_prepare_ssd_kernel<K>, smem, done)) return JIB_E_LAUNCH;
    JIB_LAUNCH((chunk_prepare_ssd_kernel<K>), dim3(a.T / C + a.n_seqs, a.H / a.rep * ((a.rep + HB - 1) / HB) + (a.H * a.V + 255) / 256), NT, smem, s, a);
    const int rc = launched();
    return rc ? rc : launch_pass<SSD, K>(a, s);
}

long long rec_bytes(const jib_state_mix & a) {
#define REC(KIND, FIELD) (a.K == 64 ? Rec<KIND, 64>::FIELD : Rec<KIND, 128>::FIELD)
    const long long nch = a.T / C + a.n_seqs;
    if (per_head(a.kind)) return nch * (a.H / a.rep * REC(SSD, A) + a.H * (REC(SSD, BYTES) - REC(SSD, A)));
    return nch * a.H * (a.kind == DELTA ? REC(DELTA, BYTES) + C * 4 * a.V : REC(LINEAR, BYTES));
#undef REC
}

}  // namespace

bool jib_state_chunk_ok(const jib_state_mix & a) {
    const long long cols = a.ld | a.q_off | a.k_off | a.v_off | a.conv0 | a.n_conv | (per_head(a.kind) ? 0 : a.ld_dec);
    if (a.kind == MLSTM && (a.q_off | a.k_off) % 8) return false;
    if ((a.kind == HGRN || a.kind == MLSTM) && (a.ld % 8 || a.v_off % 8 || a.taps != 0 || ((uintptr_t) a.proj & 15))) return false;
    return (a.K == 64 || a.K == 128) && a.V % 16 == 0 && a.V <= 256 && a.taps <= 4 && cols % 4 == 0 && ((uintptr_t) a.proj & 7) == 0 &&
           (per_head(a.kind) || ((uintptr_t) a.dec_in & 7) == 0) && a.H % a.rep == 0;
}

int jib_state_chunk_run(const jib_state_mix & a, cudaStream_t s) {
    if (rec_bytes(a) > a.chunk_bytes) return JIB_E_SCRATCH;
    switch (a.kind) {
        case DELTA: return a.K == 64 ? run_chunks<DELTA, 64>(a, s) : run_chunks<DELTA, 128>(a, s);
        case LINEAR: return a.K == 64 ? run_chunks<LINEAR, 64>(a, s) : run_chunks<LINEAR, 128>(a, s);
        case HGRN: return a.K == 64 ? run_chunks<HGRN, 64>(a, s) : run_chunks<HGRN, 128>(a, s);
        case MLSTM: return a.K == 64 ? run_chunks_mlstm<64>(a, s) : run_chunks_mlstm<128>(a, s);
        default: return a.K == 64 ? run_chunks_ssd<64>(a, s) : run_chunks_ssd<128>(a, s);
    }
}

// Bytes of scratch (m->chunk) with which jib_state_mix_run takes a batch of portions through the tensor cores; 0: not these sizes.
extern "C" JIB_EXPORT long long jib_state_chunk_bytes(const jib_state_mix * m) { return jib_state_chunk_ok(*m) ? rec_bytes(*m) : 0; }
