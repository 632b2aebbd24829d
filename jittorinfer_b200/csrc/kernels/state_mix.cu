// Token mixers with a matrix state per head: S [K key channels][V value channels], fp32, one per sequence slot and head.
//
//   S <- diag(decay_t) S;   u = s_t (v_t - [delta] S^T k_t);   S <- S + k_t u^T;   o_t = S^T q_t + D v_t
//
// in kinds that differ in where q, k, v, the decay and the factor s come from:
//   DELTA   q, k unit vectors, one decay per (head, key channel) = exp(-a_h softplus(. + bias)), s = sigmoid(.), the delta term
//   LINEAR  one decay per (head, key channel) = sigmoid(. + bias)^(1/tau), s = 1
//   SSD     one decay per head = exp(-a_h s), s = softplus(. + bias); q and k shared by a group of heads
//   HGRN    one decay f per (head, key channel), bounded from below, k = 1 - f, silu on q, s = 1
//   MLSTM   one decay per head = exp(f + m - m'), s = exp(i - m'), relative to a running maximum m' = max(f + m, i) of the log gates; a
//           vector n of keys that decays and grows like the state; o is divided by max(|n . q|, exp(-m')) + 1e-6
// A window of the projection's columns may pass a short causal convolution and silu first (DELTA: q, k, v; SSD: v, k, q).
// What follows the read-out: DELTA / LINEAR / MLSTM a norm over each head's V channels times a gate, HGRN the norm alone; SSD a gate, then a
// norm over parts of the row.
//
// Single tokens (decode): state_step does all of it in one launch per layer (SSD: plus the gated norm of whole rows).
// Portions: state_prep (convolution, unit norm, decays -> fp32; MLSTM: mlstm_gates ahead of it), state_scan (the recurrence, token by token),
// state_finish (gate and norm); bf16 portions of the head sizes it is built for take state_chunk.cu in place of the first two.
//
// A sequence's state lives in row seq_slots[b] of [n_state][H][K][V]; its last convolution inputs in a ring [n_state][taps][channels]
// whose row p % taps holds position p's.  A range that starts at position 0 starts from zeros whatever the rows hold, so slots are
// handed on without clearing.  Sequence b owns token rows q_start[b] .. q_start[b + 1].  Activations bf16 or fp32, the rest fp32.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <stdint.h>

#include "jib_kernels.h"
#include "pdl.cuh"
#include "sm100.cuh"
#include "state_mix.cuh"

namespace {

using namespace state_mix;

// ---- portions: inputs of the recurrence in fp32 ------------------------------------------------------------------------------
// qk [T][2][Hk][K], v [T][H][V], dec [T][H][K] (SSD: [T][H]), s [T][H].  One warp per (token, item); items: q heads, k heads,
// value heads, then one for the per-head factors and (DELTA, LINEAR) one per head's decays.
// MLSTM: v and o have one more column, v = 1, whose state is n.
constexpr int PREP_C = 16;                                   // channels of a q / k head per lane: K <= 32 * PREP_C

template <typename T, int KIND>
__global__ void __launch_bounds__(256) state_prep_kernel(const __grid_constant__ jib_state_mix a) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int lane = threadIdx.x & 31, t = blockIdx.y;
    const int Hk = a.H / a.rep;
    int item = blockIdx.x * 8 + (threadIdx.x >> 5);
    const int b = seq_of(a.q_start, a.n_seqs, t), back = t - a.q_start[b], p = a.positions[t];
    const int slot = a.taps > 0 ? checked_slot(a, b, 45) : -1;
    if (item < 2 * Hk) {
        const bool is_q = item < Hk;
        const int c0 = (is_q ? a.q_off : a.k_off) + (is_q ? item : item - Hk) * a.K;
        float v[PREP_C], ss = 0.f;
#pragma unroll
        for (int i = 0; i < PREP_C; ++i) {
            const int c = lane + 32 * i;
            v[i] = 0.f;
            if (c >= a.K) continue;
            if (KIND == HGRN && !is_q) {
                const int g = (item - Hk) * a.K + c;
                float f;
                bounded_gate(to_f(((const T *) a.dec_in)[(size_t) t * a.ld_dec + g]) + a.bias[g], a.lower[g], f, v[i]);
            } else {
                v[i] = column<T>(a, t, c0 + c, p, back, slot);
                if (KIND == HGRN) v[i] = silu<T>(v[i]);
            }
            if (KIND == DELTA) ss += v[i] * v[i];
        }
        float scale = is_q && KIND != MLSTM ? a.q_scale : 1.f;
        if (KIND == DELTA) scale /= sqrtf(warp_sum(ss) + 1e-6f);
        float * out = a.qk + ((size_t) t * 2 * Hk + item) * a.K;
#pragma unroll
        for (int i = 0; i < PREP_C; ++i)
            if (lane + 32 * i < a.K) out[lane + 32 * i] = v[i] * scale;
        return;
    }
    item -= 2 * Hk;
    if (item < a.H) {
        const int VS = scratch_cols(KIND, a.V);
        for (int c = lane; c < VS; c += 32)
            a.v[((size_t) t * a.H + item) * VS + c] = c < a.V ? column<T>(a, t, a.v_off + item * a.V + c, p, back, slot) : c == a.V ? 1.f : 0.f;
        return;
    }
    item -= a.H;
    if ((KIND == DELTA || KIND == SSD) && item == 0) {
        for (int h = lane; h < a.H; h += 32) {
            const float s = head_factor<KIND>(a, to_f(((const T *) a.proj)[(size_t) t * a.ld + a.s_off + h]), h);
            a.s[(size_t) t * a.H + h] = s;
            if (KIND == SSD) a.dec[(size_t) t * a.H + h] = expf(a.neg_a[h] * s);
        }
        return;
    }
    if (KIND == DELTA || KIND == SSD) --item;
    if (per_channel(KIND) && item < a.H)
        for (int c = lane; c < a.K; c += 32) {
            const int i = item * a.K + c;
            const float z = to_f(((const T *) a.dec_in)[(size_t) t * a.ld_dec + i]) + a.bias[i];
            float f, rest;
            if (KIND == HGRN) bounded_gate(z, a.lower[i], f, rest);
            else f = channel_decay<KIND>(a, z, item);
            a.dec[(size_t) t * a.H * a.K + i] = f;
        }
}

// ---- portions, MLSTM: gates relative to the running maximum --------------------------------------------------------------------
// m_t = max(f_t + m_(t-1), i_t) is a composition of maps m -> max(m + A, B).  grid (H, n_seqs): a thread composes the maps of GATE_N tokens, the
// CTA scans the compositions, then every thread runs its tokens from where it knows m.  Writes the decays (base-2 logarithms with log2), the
// factors s, the maxima, and the sequence's new maximum.
constexpr int GATE_NT = 256, GATE_N = 8;

template <typename T>
__global__ void __launch_bounds__(GATE_NT) mlstm_gates_kernel(const __grid_constant__ jib_state_mix a, int log2) {
    __shared__ float wa[GATE_NT / 32], wb[GATE_NT / 32];
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int h = blockIdx.x, b = blockIdx.y, H = a.H, warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int q0 = a.q_start[b], n = a.q_start[b + 1] - q0;
    if (n <= 0) return;
    const int slot = checked_slot(a, b, 50);
    float * top = a.extra + ((size_t) (slot < 0 ? 0 : slot) * H + h) * (a.K + 1) + a.K;
    float m0 = slot >= 0 && a.positions[q0] > 0 ? *top : 0.f;
    const float bi = a.bias[h], bf = a.bias[H + h];
    __syncthreads();                                         // read before the last token's thread replaces it
    for (int t0 = 0; t0 < n; t0 += GATE_NT * GATE_N) {
        float gi[GATE_N], gf[GATE_N], A = 0.f, B = -INFINITY;
        const int first = t0 + threadIdx.x * GATE_N;
#pragma unroll
        for (int i = 0; i < GATE_N; ++i) {
            const T * z = (const T *) a.dec_in + (size_t) (q0 + min(first + i, n - 1)) * a.ld_dec + h;
            gi[i] = to_f(z[0]) + bi;
            gf[i] = to_f(z[H]) + bf;
        }
#pragma unroll
        for (int i = 0; i < GATE_N; ++i) {
            gi[i] = first + i < n ? log_input_gate(gi[i], a.gate_cap) : -INFINITY;
            gf[i] = first + i < n ? log_forget_gate(gf[i], a.gate_cap) : 0.f;
            A += gf[i];
            B = fmaxf(B + gf[i], gi[i]);
        }
        // exclusive scan: x -> max(x + A, B) of all tokens before this thread's
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const float pa = __shfl_up_sync(0xffffffffu, A, o), pb = __shfl_up_sync(0xffffffffu, B, o);
            if (lane >= o) {
                B = fmaxf(pb + A, B);
                A += pa;
            }
        }
        if (lane == 31) {
            wa[warp] = A;
            wb[warp] = B;
        }
        A = __shfl_up_sync(0xffffffffu, A, 1);
        B = __shfl_up_sync(0xffffffffu, B, 1);
        if (lane == 0) {
            A = 0.f;
            B = -INFINITY;
        }
        __syncthreads();
        float m = m0, next = m0;
        for (int w = 0; w < GATE_NT / 32; ++w) {
            if (w < warp) m = fmaxf(m + wa[w], wb[w]);
            next = fmaxf(next + wa[w], wb[w]);
        }
        m = fmaxf(m + A, B);
#pragma unroll
        for (int i = 0; i < GATE_N; ++i) {
            if (first + i >= n) break;
            const float x = gf[i] + m, mt = fmaxf(x, gi[i]);
            const size_t at = (size_t) (q0 + first + i) * H + h;
            a.dec[at] = log2 ? (x - mt) * 1.4426950408889634f : expf(x - mt);
            a.s[at] = expf(gi[i] - mt);
            a.tops[at] = mt;
            m = mt;
            if (slot >= 0 && first + i == n - 1) *top = mt;
        }
        m0 = next;
        __syncthreads();                                     // wa, wb are free
    }
}

// ---- portions: the recurrence --------------------------------------------------------------------------------------------------
// grid (H * ceil(V / VB), n_seqs), 128 threads = VB columns of one head's state x LK lanes; a lane keeps 16 of the K channels of its
// column in registers, channels (j * LK + lane) * 4 + e.  Tokens are staged through shared memory SCAN_TT at a time, one tile
// ahead.  Also stores the range's last convolution inputs (their old values were read by state_prep).
constexpr int SCAN_NT = 128, SCAN_TT = 8;

template <typename T, int KIND, int LK>
__global__ void __launch_bounds__(SCAN_NT) state_scan_kernel(const __grid_constant__ jib_state_mix a, int splits, int aligned) {
    constexpr int KP = LK * 16, VB = SCAN_NT / LK;
    constexpr bool CHANNELS = per_channel(KIND);
    constexpr int ROW = (CHANNELS ? 3 : 2) * KP;             // k | q | decay
    constexpr int TILE = SCAN_TT * (ROW + VB + 2);
    extern __shared__ float smem[];
    PDL_TRIGGER_TOP();
    const int h = blockIdx.x / splits, v0 = (blockIdx.x % splits) * VB;
    const int b = blockIdx.y, lane = threadIdx.x % LK, col = threadIdx.x / LK;
    const int K = a.K, V = a.V, H = a.H, Hk = H / a.rep, VS = scratch_cols(KIND, V), nv = min(VB, V + (KIND == MLSTM) - v0);
    for (int i = threadIdx.x; i < 2 * TILE; i += SCAN_NT) smem[i] = 0.f;       // channels past K stay zero
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int q0 = a.q_start[b], n = a.q_start[b + 1] - q0;
    if (n <= 0) return;
    const int slot = checked_slot(a, b, 46);
    store_conv_tail<T>(a, slot, q0, n, blockIdx.x * SCAN_NT + threadIdx.x, gridDim.x * SCAN_NT);
    const bool mine = col < nv, sum = KIND == MLSTM && v0 + col == V;
    const size_t at = (size_t) (slot < 0 ? 0 : slot) * H + h, ld = sum ? 1 : V;
    float * st = sum ? a.extra + at * (K + 1) : a.state + at * K * V + v0 + col;
    float s[16];
    const bool past = slot >= 0 && a.positions[q0] > 0;
#pragma unroll
    for (int i = 0; i < 16; ++i) {
        const int c = ((i >> 2) * LK + lane) * 4 + (i & 3);
        s[i] = past && mine && c < K ? st[c * ld] : 0.f;
    }
    const float * kp = a.qk + ((size_t) q0 * 2 * Hk + Hk + h / a.rep) * K;
    const float * qp = a.qk + ((size_t) q0 * 2 * Hk + h / a.rep) * K;
    const float * vp = a.v + ((size_t) q0 * H + h) * VS + v0;
    const float * dp = a.dec + (CHANNELS ? ((size_t) q0 * H + h) * K : (size_t) q0 * H + h);
    const float * sp = a.s + (size_t) q0 * H + h;
    auto stage = [&](int t0, float * d) {
        const int m = min(SCAN_TT, n - t0);
        constexpr int NR = CHANNELS ? 3 : 2;
        if (aligned) {
            const int k4 = K / 4;
            for (int i = threadIdx.x; i < m * NR * k4; i += SCAN_NT) {
                const int c = i % k4, r = i / k4, tok = r / NR, w = r - tok * NR;
                const size_t row = t0 + tok;
                const float * src = w == 0 ? kp + row * 2 * Hk * K : w == 1 ? qp + row * 2 * Hk * K : dp + row * H * K;
                cp16(d + tok * ROW + w * KP + 4 * c, src + 4 * c);
            }
        } else {
            for (int i = threadIdx.x; i < m * NR * K; i += SCAN_NT) {
                const int c = i % K, r = i / K, tok = r / NR, w = r - tok * NR;
                const size_t row = t0 + tok;
                const float * src = w == 0 ? kp + row * 2 * Hk * K : w == 1 ? qp + row * 2 * Hk * K : dp + row * H * K;
                cp4(d + tok * ROW + w * KP + c, src + c);
            }
        }
        float * dv = d + SCAN_TT * ROW;
        for (int i = threadIdx.x; i < m * nv; i += SCAN_NT) cp4(dv + (i / nv) * VB + i % nv, vp + (size_t) (t0 + i / nv) * H * VS + i % nv);
        float * ds = dv + SCAN_TT * VB;
        if (threadIdx.x < m) {
            if (KIND == DELTA || !CHANNELS) cp4(ds + threadIdx.x, sp + (size_t) (t0 + threadIdx.x) * H);
            if (!CHANNELS) cp4(ds + SCAN_TT + threadIdx.x, dp + (size_t) (t0 + threadIdx.x) * H);
        }
        asm volatile("cp.async.commit_group;" ::: "memory");
    };
    __syncthreads();
    stage(0, smem);
    const float skip = KIND == SSD ? a.skip[h] : 0.f;
    float * op = a.o + ((size_t) q0 * H + h) * VS + v0 + col;
    int buf = 0;
    for (int t0 = 0; t0 < n; t0 += SCAN_TT, buf ^= 1) {
        if (t0 + SCAN_TT < n) {
            stage(t0 + SCAN_TT, smem + (buf ^ 1) * TILE);
            asm volatile("cp.async.wait_group 1;" ::: "memory");
        } else {
            asm volatile("cp.async.wait_group 0;" ::: "memory");
        }
        __syncthreads();
        const float * d = smem + buf * TILE;
        const float * dv = d + SCAN_TT * ROW, * ds = dv + SCAN_TT * VB;
        const int m = min(SCAN_TT, n - t0);
        for (int i = 0; i < m; ++i) {
            float k[16], q[16];
            const float * row = d + i * ROW + 4 * lane;
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const float4 x = *(const float4 *) (row + 4 * LK * j), y = *(const float4 *) (row + KP + 4 * LK * j);
                k[4 * j] = x.x; k[4 * j + 1] = x.y; k[4 * j + 2] = x.z; k[4 * j + 3] = x.w;
                q[4 * j] = y.x; q[4 * j + 1] = y.y; q[4 * j + 2] = y.z; q[4 * j + 3] = y.w;
            }
            if (!CHANNELS) {
                const float g = ds[SCAN_TT + i];
#pragma unroll
                for (int c = 0; c < 16; ++c) s[c] *= g;
            } else {
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const float4 g = *(const float4 *) (row + 2 * KP + 4 * LK * j);
                    s[4 * j] *= g.x; s[4 * j + 1] *= g.y; s[4 * j + 2] *= g.z; s[4 * j + 3] *= g.w;
                }
            }
            const float v = dv[i * VB + col];
            float u = v;
            if (KIND == DELTA) {
                float e[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
                for (int c = 0; c < 16; ++c) e[c & 3] += s[c] * k[c];
                float r = (e[0] + e[1]) + (e[2] + e[3]);
#pragma unroll
                for (int o = LK / 2; o > 0; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
                u = v - r;
            }
            if (KIND == DELTA || !CHANNELS) u *= ds[i];
            float e[4] = {0.f, 0.f, 0.f, 0.f};
#pragma unroll
            for (int c = 0; c < 16; ++c) {
                s[c] += k[c] * u;
                e[c & 3] += s[c] * q[c];
            }
            float r = (e[0] + e[1]) + (e[2] + e[3]);
#pragma unroll
            for (int o = LK / 2; o > 0; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
            if (lane == 0 && mine) op[(size_t) (t0 + i) * H * VS] = KIND == SSD ? r + skip * v : r;
        }
        __syncthreads();
    }
    if (slot >= 0 && mine) {
#pragma unroll
        for (int i = 0; i < 16; ++i) {
            const int c = ((i >> 2) * LK + lane) * 4 + (i & 3);
            if (c < K) st[c * ld] = s[i];
        }
    }
}

// ---- gate and norm of the read-out ---------------------------------------------------------------------------------------------
// Vectors of E adjacent values (E 4 or 1: rows of any size and alignment).
template <int E> struct Vals { float v[E]; };
template <int E> __device__ __forceinline__ Vals<E> load_vals(const float * p) {
    Vals<E> r;
    if (E == 4) *(float4 *) r.v = *(const float4 *) p;
    else r.v[0] = *p;
    return r;
}
template <int E> __device__ __forceinline__ Vals<E> load_vals(const bf16 * p) {
    Vals<E> r;
    if (E == 4) {
        const uint2 x = *(const uint2 *) p;
        const float2 a = __bfloat1622float2(*(const __nv_bfloat162 *) &x.x), b = __bfloat1622float2(*(const __nv_bfloat162 *) &x.y);
        r.v[0] = a.x; r.v[1 % E] = a.y; r.v[2 % E] = b.x; r.v[3 % E] = b.y;
    } else {
        r.v[0] = to_f(*p);
    }
    return r;
}
template <int E> __device__ __forceinline__ void store_vals(float * p, const Vals<E> & r) {
    if (E == 4) *(float4 *) p = *(const float4 *) r.v;
    else *p = r.v[0];
}
template <int E> __device__ __forceinline__ void store_vals(bf16 * p, const Vals<E> & r) {
    if (E == 4) {
        uint2 x;
        *(__nv_bfloat162 *) &x.x = __floats2bfloat162_rn(r.v[0], r.v[1 % E]);
        *(__nv_bfloat162 *) &x.y = __floats2bfloat162_rn(r.v[2 % E], r.v[3 % E]);
        *(uint2 *) p = x;
    } else {
        put(p, r.v[0]);
    }
}

// All but SSD: one warp per (token, head): o / rms(o) * norm_w [* gate]; MLSTM: o is divided by its size first.  V <= 32 * N * E.
template <typename T, int KIND, int E, int N>
__global__ void __launch_bounds__(256) state_finish_kernel(const __grid_constant__ jib_state_mix a) {
    PDL_TRIGGER_TOP();
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int lane = threadIdx.x & 31, i = blockIdx.x * 8 + (threadIdx.x >> 5), t = i / a.H, h = i % a.H, V = a.V;
    if (t >= a.T) return;
    const float * o = a.o + (size_t) i * scratch_cols(KIND, V), * norm_w = a.norm_w + (KIND == MLSTM ? h * V : 0);
    const T * gate = (const T *) a.gate + (size_t) t * a.ld_gate + h * V;
    T * y = (T *) a.y + (size_t) t * a.ldy + h * V;
    const float size = KIND == MLSTM ? a.q_scale / (fmaxf(fabsf(o[V] * a.q_scale), expf(-a.tops[i])) + 1e-6f) : 1.f;
    Vals<E> x[N], g[N], w[N];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < N; ++k) {                            // everything the row needs is requested before any of it is used
        const int c = (lane + 32 * k) * E;
        if (c >= V) continue;
        x[k] = load_vals<E>(o + c);
        if (KIND != HGRN) g[k] = load_vals<E>(gate + c);
        w[k] = load_vals<E>(norm_w + c);
    }
#pragma unroll
    for (int k = 0; k < N; ++k)
        if ((lane + 32 * k) * E < V)
#pragma unroll
            for (int e = 0; e < E; ++e) {
                if (KIND == MLSTM) x[k].v[e] *= size;
                ss += x[k].v[e] * x[k].v[e];
            }
    const float inv = a.out_scale * rsqrtf(warp_sum(ss) / (float) V + a.eps);
#pragma unroll
    for (int k = 0; k < N; ++k) {
        const int c = (lane + 32 * k) * E;
        if (c >= V) continue;
#pragma unroll
        for (int e = 0; e < E; ++e)
            x[k].v[e] *= inv * w[k].v[e] * (KIND == HGRN ? 1.f : KIND == LINEAR ? silu<T>(g[k].v[e]) : sigmoid<T>(g[k].v[e]));
        store_vals<E>(y + c, x[k]);
    }
}

// SSD: one CTA per (token, part of the row): y = o * silu(gate), then y / rms(y) * norm_w over the part.
template <typename T, int E>
__global__ void __launch_bounds__(256) state_gate_norm_kernel(const __grid_constant__ jib_state_mix a) {
    PDL_TRIGGER_TOP();
    __shared__ float red[8];
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    const int t = blockIdx.y, inner = a.H * a.V, m = inner / a.norm_groups, c0 = blockIdx.x * m;
    const float * o = a.o + (size_t) t * inner + c0, * w = a.norm_w + c0;
    const T * gate = (const T *) a.gate + (size_t) t * a.ld_gate + c0;
    T * y = (T *) a.y + (size_t) t * a.ldy + c0;
    constexpr int KEEP = 4;                                  // vectors a thread holds; longer parts are computed twice
    Vals<E> v[KEEP], g[KEEP];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int c = (threadIdx.x + 256 * i) * E;
        if (c >= m) continue;
        v[i] = load_vals<E>(o + c);
        g[i] = load_vals<E>(gate + c);
    }
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        if ((threadIdx.x + 256 * i) * E >= m) continue;
#pragma unroll
        for (int e = 0; e < E; ++e) {
            v[i].v[e] *= silu<T>(g[i].v[e]);
            ss += v[i].v[e] * v[i].v[e];
        }
    }
    for (int c = (threadIdx.x + 256 * KEEP) * E; c < m; c += 256 * E)
        for (int e = 0; e < E; ++e) {
            const float x = o[c + e] * silu<T>(to_f(gate[c + e]));
            ss += x * x;
        }
    ss = warp_sum(ss);
    if ((threadIdx.x & 31) == 0) red[threadIdx.x >> 5] = ss;
    __syncthreads();
    ss = 0.f;
#pragma unroll
    for (int i = 0; i < 8; ++i) ss += red[i];
    const float inv = a.out_scale * rsqrtf(ss / (float) m + a.eps);
#pragma unroll
    for (int i = 0; i < KEEP; ++i) {
        const int c = (threadIdx.x + 256 * i) * E;
        if (c >= m) continue;
        const Vals<E> n = load_vals<E>(w + c);
#pragma unroll
        for (int e = 0; e < E; ++e) v[i].v[e] *= inv * n.v[e];
        store_vals<E>(y + c, v[i]);
    }
    for (int c = (threadIdx.x + 256 * KEEP) * E; c < m; c += 256 * E)
        for (int e = 0; e < E; ++e) put(y + c + e, o[c + e] * silu<T>(to_f(gate[c + e])) * inv * w[c + e]);
}

// ---- single tokens -------------------------------------------------------------------------------------------------------------
// grid (H, n_seqs): one CTA per head and sequence; thread = VEC adjacent columns x every NRG-th row of S, up to R rows in registers
// (KEEP: all of them, the state is read once).

template <int VEC> struct Cols { float v[VEC]; };
template <int VEC> __device__ __forceinline__ Cols<VEC> ld_cols(const float * p) {
    Cols<VEC> r;
    if (VEC == 4) *(float4 *) r.v = *(const float4 *) p;
    else r.v[0] = *p;
    return r;
}
template <int VEC> __device__ __forceinline__ void st_cols(float * p, const Cols<VEC> & c) {
    if (VEC == 4) *(float4 *) p = *(const float4 *) c.v;
    else *p = c.v[0];
}

template <typename T, int KIND, int VEC, int R, bool KEEP>
__global__ void __launch_bounds__(512, R <= 8 ? 2 : 1) state_step_kernel(const __grid_constant__ jib_state_mix a) {
    extern __shared__ float smem[];
    PDL_TRIGGER_TOP();
    const int h = blockIdx.x, t = blockIdx.y, tid = threadIdx.x, NT = blockDim.x;
    const int K = a.K, V = a.V, H = a.H;
    const int ncg = (V + VEC - 1) / VEC, nrg = NT / ncg, cg = tid % ncg, rg = tid / ncg;
    const bool live = rg < nrg;
    float * sq = smem, * sk = sq + K, * sd = sk + K, * sv = sd + K, * red = sv + (V + 3) / 4 * 4, * sums = red + nrg * ncg * VEC;
    pdl_wait();      // inputs come from earlier kernels; nothing is written before this point
    int slot = a.seq_slots[t];
    if (slot >= a.n_state) {
        if (h == 0 && tid == 0) jib_report(a.status, JIB_ERR_BOUNDS, 47, slot);
        slot = -1;
    }
    const int p = a.positions[t];
    const bool past = slot >= 0 && p > 0;
    float * st = a.state + ((size_t) (slot < 0 ? 0 : slot) * H + h) * K * V + cg * VEC;
    Cols<VEC> s[R];                                          // R rows
    auto load = [&](int r0) {
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int r = r0 + rg + i * nrg;
            if (past && live && r < K) {
                s[i] = ld_cols<VEC>(st + (size_t) r * V);
            } else {
#pragma unroll
                for (int e = 0; e < VEC; ++e) s[i].v[e] = 0.f;
            }
        }
    };
    if (KEEP) load(0);                                       // in flight while the inputs are prepared
    const int hk = h / a.rep;
    float n_old[KIND == MLSTM ? 2 : 1];                      // MLSTM: what the keys add up to, K <= 512 on 256 threads or more
    float * const extra = KIND == MLSTM ? a.extra + ((size_t) (slot < 0 ? 0 : slot) * H + h) * (K + 1) : nullptr;
    float top = 0.f;
    if (KIND == MLSTM) {
#pragma unroll
        for (int j = 0; j < 2; ++j) n_old[j % (KIND == MLSTM ? 2 : 1)] = past && tid + j * NT < K ? extra[tid + j * NT] : 0.f;
        if (past) top = extra[K];
    }
    for (int i = tid; i < (per_channel(KIND) ? 3 : 2) * K + V; i += NT) {
        if (i < K) sq[i] = KIND == HGRN ? silu<T>(column_single<T>(a, t, a.q_off + hk * K + i, p, slot)) : column_single<T>(a, t, a.q_off + hk * K + i, p, slot);
        else if (i < 2 * K && KIND == HGRN) continue;        // comes with the decay
        else if (i < 2 * K) sk[i - K] = column_single<T>(a, t, a.k_off + hk * K + i - K, p, slot);
        else if (i < 2 * K + V) sv[i - 2 * K] = column_single<T>(a, t, a.v_off + h * V + i - 2 * K, p, slot);
        else {
            const int c = i - 2 * K - V, g = h * K + c;
            const float z = to_f(((const T *) a.dec_in)[(size_t) t * a.ld_dec + g]) + a.bias[g];
            if (KIND == HGRN) bounded_gate(z, a.lower[g], sd[c], sk[c]);
            else sd[c] = channel_decay<KIND>(a, z, h);
        }
    }
    float factor = 1.f, decay = 1.f;
    if (KIND == MLSTM) {
        const T * z = (const T *) a.dec_in + (size_t) t * a.ld_dec + h;
        const float gi = log_input_gate(to_f(z[0]) + a.bias[h], a.gate_cap), x = log_forget_gate(to_f(z[H]) + a.bias[H + h], a.gate_cap) + top;
        top = fmaxf(x, gi);
        decay = expf(x - top);
        factor = expf(gi - top);
    }
    if (KIND == DELTA || KIND == SSD) factor = head_factor<KIND>(a, to_f(((const T *) a.proj)[(size_t) t * a.ld + a.s_off + h]), h);
    if (KIND == SSD) decay = expf(a.neg_a[h] * factor);
    __syncthreads();
    if (a.taps > 1 && slot >= 0) {                           // this position's convolution inputs; no reader of this launch needs the row
        T * ring = (T *) a.conv_state + ((size_t) slot * a.taps + p % a.taps) * a.n_conv;
        const T * x = (const T *) a.proj + (size_t) t * a.ld;
        const bool owner = h % a.rep == 0;
        for (int i = tid; i < (owner ? 2 * K : 0) + V; i += NT) {
            const int c = i < V ? a.v_off + h * V + i : (i < V + K ? a.q_off + hk * K + i - V : a.k_off + hk * K + i - V - K);
            ring[c - a.conv0] = x[c];
        }
    }
    float qn = a.q_scale, kn = 1.f;
    if (KIND == MLSTM) {                                     // n, and its product with q
        float d = 0.f;
#pragma unroll
        for (int j = 0; j < 2; ++j) {
            const int c = tid + j * NT;
            if (c >= K) continue;
            const float x = n_old[j % (KIND == MLSTM ? 2 : 1)] * decay + factor * sk[c];
            d += x * sq[c];
            if (slot >= 0) extra[c] = x;
        }
        if (slot >= 0 && tid == 0) extra[K] = top;           // read by all threads ahead of the barrier above
        d = warp_sum(d);
        if ((tid & 31) == 0) sums[2 + NT / 32 + (tid >> 5)] = d;
    }
    if (KIND == DELTA) {
        if (tid < 64) {
            const float * x = tid < 32 ? sq : sk;
            float ss = 0.f;
            for (int c = tid & 31; c < K; c += 32) ss += x[c] * x[c];
            ss = warp_sum(ss);
            if ((tid & 31) == 0) sums[tid >> 5] = 1.f / sqrtf(ss + 1e-6f);
        }
        __syncthreads();
        qn *= sums[0];
        kn = sums[1];
        // S^T k after the decay
        Cols<VEC> d;
#pragma unroll
        for (int e = 0; e < VEC; ++e) d.v[e] = 0.f;
        for (int r0 = 0; r0 < K; r0 += nrg * R) {
            if (!KEEP) load(r0);
#pragma unroll
            for (int i = 0; i < R; ++i) {
                const int r = r0 + rg + i * nrg;
                if (r >= K) continue;
                const float g = sd[r], kk = sk[r] * kn;
#pragma unroll
                for (int e = 0; e < VEC; ++e) d.v[e] += s[i].v[e] * g * kk;
            }
        }
        if (live) st_cols<VEC>(red + (rg * ncg + cg) * VEC, d);
        __syncthreads();
    }
    Cols<VEC> u, o;
#pragma unroll
    for (int e = 0; e < VEC; ++e) {
        o.v[e] = 0.f;
        u.v[e] = live && cg * VEC + e < V ? sv[cg * VEC + e] : 0.f;
    }
    if (KIND == DELTA && live)
        for (int g = 0; g < nrg; ++g) {
            const Cols<VEC> d = ld_cols<VEC>(red + (g * ncg + cg) * VEC);
#pragma unroll
            for (int e = 0; e < VEC; ++e) u.v[e] -= d.v[e];
        }
#pragma unroll
    for (int e = 0; e < VEC; ++e) u.v[e] *= factor * kn;
    for (int r0 = 0; r0 < K; r0 += nrg * R) {
        if (!KEEP) load(r0);
#pragma unroll
        for (int i = 0; i < R; ++i) {
            const int r = r0 + rg + i * nrg;
            if (r >= K || !live) continue;
            const float g = per_channel(KIND) ? sd[r] : decay, kk = sk[r], qq = sq[r];
#pragma unroll
            for (int e = 0; e < VEC; ++e) {
                s[i].v[e] = s[i].v[e] * g + kk * u.v[e];
                o.v[e] += s[i].v[e] * qq;
            }
            if (slot >= 0) st_cols<VEC>(st + (size_t) r * V, s[i]);
        }
    }
    if (KIND == DELTA) __syncthreads();                      // red is read above
    if (live) st_cols<VEC>(red + (rg * ncg + cg) * VEC, o);
    __syncthreads();
    // columns back to one thread each: sum over the row groups, then norm and gate
    float ss = 0.f;
    for (int c = tid; c < V; c += NT) {
        float v = 0.f;
        for (int g = 0; g < nrg; ++g) v += red[g * ncg * VEC + c];
        v *= qn;
        if (KIND == SSD) a.o[((size_t) t * H + h) * V + c] = v + a.skip[h] * sv[c];
        else sv[c] = v;
        ss += v * v;
    }
    if (KIND == SSD) return;
    ss = warp_sum(ss);
    if ((tid & 31) == 0) sums[2 + (tid >> 5)] = ss;
    __syncthreads();
    ss = 0.f;
    for (int i = 0; i < NT / 32; ++i) ss += sums[2 + i];
    float size = 1.f;
    if (KIND == MLSTM) {
        float d = 0.f;
        for (int i = 0; i < NT / 32; ++i) d += sums[2 + NT / 32 + i];
        size = 1.f / (fmaxf(fabsf(d * qn), expf(-top)) + 1e-6f);
    }
    const float inv = a.out_scale * size * rsqrtf(ss * size * size / (float) V + a.eps);
    const T * gate = (const T *) a.gate + (size_t) t * a.ld_gate + h * V;
    const float * norm_w = a.norm_w + (KIND == MLSTM ? h * V : 0);
    T * y = (T *) a.y + (size_t) t * a.ldy + h * V;
    for (int c = tid; c < V; c += NT) {
        const float g = KIND == HGRN ? 0.f : to_f(gate[c]);
        put(y + c, sv[c] * inv * norm_w[c] * (KIND == HGRN ? 1.f : KIND == LINEAR ? silu<T>(g) : sigmoid<T>(g)));
    }
}

inline int launched() { return cudaGetLastError() == cudaSuccess ? 0 : JIB_E_LAUNCH; }

template <typename T, int KIND, int LK>
int launch_scan(const jib_state_mix & a, cudaStream_t s) {
    constexpr int VB = SCAN_NT / LK, SMEM = 2 * SCAN_TT * ((per_channel(KIND) ? 3 : 2) * LK * 16 + VB + 2) * 4;
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    if (!jib::ensure_dyn_smem(state_scan_kernel<T, KIND, LK>, SMEM, done)) return JIB_E_LAUNCH;
    const int splits = (a.V + (KIND == MLSTM) + VB - 1) / VB;
    // a plain launch: as a programmatic dependent its CTAs would settle wherever the last CTAs of state_prep leave room, several to an SM
    state_scan_kernel<T, KIND, LK><<<dim3(a.H * splits, a.n_seqs), SCAN_NT, SMEM, s>>>(a, splits, a.K % 4 == 0);
    return launched();
}

template <typename T, int KIND>
int launch_finish(const jib_state_mix & a, cudaStream_t s) {
    const int part = KIND == SSD ? a.H * a.V / a.norm_groups : a.V;
    const bool vec = part % 4 == 0 && a.ld_gate % 4 == 0 && a.ldy % 4 == 0 && (((uintptr_t) a.gate | (uintptr_t) a.y) & (4 * sizeof(T) - 1)) == 0;
    if (KIND == SSD) {
        if (vec) JIB_LAUNCH((state_gate_norm_kernel<T, 4>), dim3(a.norm_groups, a.T), 256, 0, s, a);
        else JIB_LAUNCH((state_gate_norm_kernel<T, 1>), dim3(a.norm_groups, a.T), 256, 0, s, a);
    } else {
        const long long items = (long long) a.H * a.T;
        const dim3 grid((unsigned) ((items + 7) / 8));
        if (vec && a.V <= 128) JIB_LAUNCH((state_finish_kernel<T, KIND, 4, 1>), grid, 256, 0, s, a);
        else if (vec && a.V <= 512) JIB_LAUNCH((state_finish_kernel<T, KIND, 4, 4>), grid, 256, 0, s, a);
        else if (a.V <= 512) JIB_LAUNCH((state_finish_kernel<T, KIND, 1, 16>), grid, 256, 0, s, a);
        else return JIB_E_ARG;
    }
    return launched();
}

template <typename T, int KIND, int VEC, int R, bool KEEP>
int launch_step(const jib_state_mix & a, int nt, cudaStream_t s) {
    const int ncg = (a.V + VEC - 1) / VEC, nrg = nt / ncg;
    const int smem = (3 * a.K + (a.V + 3) / 4 * 4 + nrg * ncg * VEC + 2 + 32) * 4;      // sums: 2 + at most 2 per warp
    static std::atomic<unsigned char> done[jib::MAX_DEVICES];
    if (smem > 100 * 1024 || !jib::ensure_dyn_smem(state_step_kernel<T, KIND, VEC, R, KEEP>, 100 * 1024, done)) return JIB_E_ARG;
    JIB_LAUNCH((state_step_kernel<T, KIND, VEC, R, KEEP>), dim3(a.H, a.n_seqs), nt, smem, s, a);
    return KIND == SSD ? launch_finish<T, SSD>(a, s) : launched();
}
template <typename T, int KIND, int VEC>
int step(const jib_state_mix & a, cudaStream_t s) {
    const int ncg = (a.V + VEC - 1) / VEC;
    if (ncg > 512) return JIB_E_ARG;
    const int nt = ncg > 256 || (long long) a.K * a.V >= 16384 ? 512 : 256, rows = nt / ncg;
    if (rows * 4 >= a.K) return launch_step<T, KIND, VEC, 4, true>(a, nt, s);
    if (rows * 8 >= a.K) return launch_step<T, KIND, VEC, 8, true>(a, nt, s);
    if (rows * 16 >= a.K) return launch_step<T, KIND, VEC, 16, true>(a, nt, s);
    return launch_step<T, KIND, VEC, 8, false>(a, nt, s);
}

template <typename T, int KIND>
int run(const jib_state_mix & a, int single, cudaStream_t s) {
    if (single) {
        return a.V % 4 == 0 && a.K % 4 == 0 ? step<T, KIND, 4>(a, s) : step<T, KIND, 1>(a, s);
    }
    const bool chunks = sizeof(T) == 2 && a.chunk != nullptr && jib_state_chunk_ok(a);
    if (KIND == MLSTM) {
        JIB_LAUNCH((mlstm_gates_kernel<T>), dim3(a.H, a.n_seqs), GATE_NT, 0, s, a, chunks ? 1 : 0);
        const int rc = launched();
        if (rc) return rc;
    }
    if (chunks) {
        const int rc = jib_state_chunk_run(a, s);
        return rc ? rc : launch_finish<T, KIND>(a, s);
    }
    const int items = 2 * (a.H / a.rep) + a.H + (KIND == DELTA || KIND == SSD ? 1 : 0) + (per_channel(KIND) ? a.H : 0);
    JIB_LAUNCH((state_prep_kernel<T, KIND>), dim3((items + 7) / 8, a.T), 256, 0, s, a);
    int rc = launched();
    if (rc) return rc;
    if (a.K <= 16) rc = launch_scan<T, KIND, 1>(a, s);
    else if (a.K <= 32) rc = launch_scan<T, KIND, 2>(a, s);
    else if (a.K <= 64) rc = launch_scan<T, KIND, 4>(a, s);
    else if (a.K <= 128) rc = launch_scan<T, KIND, 8>(a, s);
    else if (a.K <= 256) rc = launch_scan<T, KIND, 16>(a, s);
    else rc = launch_scan<T, KIND, 32>(a, s);
    return rc ? rc : launch_finish<T, KIND>(a, s);
}

}  // namespace

extern "C" JIB_EXPORT int jib_state_mix_run(const jib_state_mix * m, int single, int f32, void * stream) {
    const jib_state_mix & a = *m;
    if (a.T <= 0 || a.n_seqs <= 0) return 0;
    if (a.H < 1 || a.K < 1 || a.V < 1 || a.K > 32 * PREP_C || a.rep < 1 || a.H % a.rep || a.T > 65535 || a.n_seqs > 65535 ||
        (a.taps > 0 && (a.conv_state == nullptr || a.conv_w == nullptr)) || (a.kind == SSD && (a.norm_groups < 1 || (a.H * a.V) % a.norm_groups)) ||
        (single && a.n_seqs != a.T) || (!single && a.chunk == nullptr && (a.qk == nullptr || a.v == nullptr || a.dec == nullptr)) ||
        ((a.kind == DELTA || a.kind == SSD) && !single && a.chunk == nullptr && a.s == nullptr) || ((a.kind == SSD || !single) && a.o == nullptr) ||
        (a.kind == HGRN && (a.lower == nullptr || a.rep != 1)) ||
        (a.kind == MLSTM && (a.extra == nullptr || a.rep != 1 || a.gate_cap <= 0.f || (!single && (a.dec == nullptr || a.s == nullptr || a.tops == nullptr)))))
        return JIB_E_ARG;
    cudaStream_t s = (cudaStream_t) stream;
    switch (a.kind) {
        case DELTA: return f32 ? run<float, DELTA>(a, single, s) : run<bf16, DELTA>(a, single, s);
        case LINEAR: return f32 ? run<float, LINEAR>(a, single, s) : run<bf16, LINEAR>(a, single, s);
        case SSD: return f32 ? run<float, SSD>(a, single, s) : run<bf16, SSD>(a, single, s);
        case HGRN: return f32 ? run<float, HGRN>(a, single, s) : run<bf16, HGRN>(a, single, s);
        case MLSTM: return f32 ? run<float, MLSTM>(a, single, s) : run<bf16, MLSTM>(a, single, s);
    }
    return JIB_E_ARG;
}
