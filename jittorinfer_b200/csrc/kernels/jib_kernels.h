// C ABI of libjib200_kernels.so: every launcher takes raw device pointers and a CUDA stream, returns
// 0 on success or a negative JIB_E_* code, and never allocates or synchronises.
#pragma once
#include <stddef.h>
#include <stdint.h>

#define JIB_EXPORT __attribute__((visibility("default")))

enum {
    JIB_E_ARG = -1,         // unsupported shape / argument
    JIB_E_ALIGN = -2,       // pointer or stride not 16-byte aligned (TMA requirement)
    JIB_E_DRIVER = -3,      // cuTensorMapEncodeTiled entry point unavailable
    JIB_E_TENSORMAP = -4,   // tensor-map encode failed
    JIB_E_LAUNCH = -5,      // kernel launch failed
    JIB_E_SCRATCH = -6,     // scratch / counter buffer too small for the requested split
};

// Activation of a gated pair: z * sigmoid(z), or 0.5 z (1 + tanh(sqrt(2 / pi) (z + 0.044715 z^3))).
enum { JIB_ACT_SILU = 0, JIB_ACT_GELU_TANH = 1 };
// Function of a single product (no w2): none, max(y, 0)^2, s y with s = scale, capped to softcap tanh(s y / softcap) unless softcap is 0, or
// gelu(r y) = r y (1 + erf(r y / sqrt 2)) / 2 with r = row_scale[row] (1 without).
enum { JIB_UNARY_NONE = 0, JIB_UNARY_RELU2 = 1, JIB_UNARY_CAP = 2, JIB_UNARY_GELU = 3 };

#ifdef __cplusplus
extern "C" {
#endif

// Y[b][t][n] = sum_k X[b][t][k] * W[b][n][k]  (bf16 in, fp32 accumulate), optional second weight
// (w2: out = act(X W^T) * (X W2^T), act = silu or the tanh form of gelu) or a function of the single product, optional residual add
// (row stride 0: one row for all tokens, i.e. a bias), optional expert-grouped rows.
typedef struct jib_gemm_desc {
    const void * x;            // bf16 activations
    const void * w;            // bf16 weights [batch][N][K]
    const void * w2;           // NULL, or second weight of the gated pair (same layout as w)
    void * out;
    const void * residual;     // NULL or [rows][N] added in the epilogue
    const int * seg;           // NULL, or device int[batch+1]: rows of expert b are [seg[b], seg[b+1]) of x / out
    void * scratch;            // split-K partials (fp32), may be NULL (then no split)
    int * counters;            // split-K tile counters, zero-initialised once; the kernel leaves them zero
    int * status;              // 4 ints, see sm100.cuh; may be NULL
    long long x_row_stride, x_batch_stride;   // elements
    long long w_row_stride, w_batch_stride;
    long long ldo, out_batch_stride, ldr, res_batch_stride;
    long long x_rows_total;    // grouped: total rows of x (all experts)
    size_t scratch_bytes;
    int n_counters;
    int T, N, K, batch;        // grouped: T = upper bound of rows of one expert
    int max_rows;              // grouped: tighter bound of rows per expert if known (else 0)
    int active_hint;           // grouped: expected number of non-empty experts (split-K heuristic), else 0
    int out_f32, res_f32;
    int splits;                // 0 = choose
    int bn;                    // 0 = choose; token-tile width 16/32/64/128/256
    int sm_count;
    int ar_site;               // fused all-reduce: call-site index (see comm_fused.cu)
    const void * ar;           // NULL, or a JibArCtx: the epilogue sums the tile over all ranks through peer memory
    const void * out_row_ptr;  // NULL, or device array [rows] of bf16 row addresses (may be peer memory): row i of the result is
                               // stored there instead of out + i * ldo (a NULL entry drops the row)
    const void * ag_flags;     // NULL, or device unsigned[ag_world]: rows [s*ag_rows, (s+1)*ag_rows) of x are valid once
    const void * ag_epoch;     //   ag_flags[s] == *ag_epoch (all-gather fused into the activation loads)
    int ag_rows, ag_world;
    int ar_rs_rows;            // with ar: > 0 = reduce-scatter by token rows (row i delivered to rank i / ar_rs_rows only)
    const int * src_token;     // grouped, small batches: x is NOT expert-sorted but holds the src_rows token rows themselves; every
    int src_rows;              //   non-empty expert multiplies all of them (src_rows <= the token tile) and result row i (in the
                               //   expert-sorted order that seg describes) is the accumulator column src_token[i]: the gather of
                               //   token rows into sorted order is never materialised
    const int * expert_list;   // grouped: NULL, or device int[n_slots]: the launch covers only these experts (entries < 0 are unused
    int n_slots;               //   slots); n_slots <= batch.  For batches that hit few experts: most of the grid would exit at once
    int list_tiles;            // 1: expert_list entries are (token tile << 16 | expert) pairs (jib_moe_tile_list, built for this bn):
                               //   the launch covers exactly the token tiles that exist instead of T / bn tiles for every expert
    int pdl_flags;             // grouped, two launches back to back over one segment table: 1 on the first (it lets its dependents
                               //   start only once the table is known to be complete), 2 on the second (it may read the table and
                               //   request weights before the first launch has finished); 0 otherwise
    int act;                   // with w2: JIB_ACT_*
    int unary;                // without w2: JIB_UNARY_*, applied before the residual (not with ar)
    float scale, softcap;     // of JIB_UNARY_CAP
    const float * row_scale;  // of JIB_UNARY_GELU: NULL, or [rows of out], a factor of each (grouped: expert-sorted) row's product
} jib_gemm_desc;

JIB_EXPORT int jib_gemm_bf16(const jib_gemm_desc * d, void * stream);
// The same product on CUDA cores (gemm_simt.cu): fp32 operands (f32 = 1, result fp32), or bf16 operands TMA cannot address.
JIB_EXPORT int jib_gemm_simt(const jib_gemm_desc * d, int f32, void * stream);

// ---- sampling (sampling.cu) ---------------------------------------------------------------------
// One id per row from the row's top-k candidates (vals / ids [n][k], sorted by value, descending; k <= 128).
// params [n][5] fp32: temperature (<= 0: best candidate), top_k (<= 0: all), top_p (>= 1: off), min_p (<= 0: off), u in [0, 1).
JIB_EXPORT int jib_sample_topk(const float * vals, const int * ids, const float * params, int * out, int n, int k, void * stream);

// Block-quantised checkpoint data (ggml types Q4_0 .. Q8_K) -> bf16, at load time (dequant.cu).
JIB_EXPORT int jib_dequantize_bf16(unsigned ggml_type, const void * src, unsigned long long n_elements, void * dst, void * stream);

// ---- memory-bound kernels (elementwise.cu) ----------------------------------------------------
JIB_EXPORT int jib_embed_gather(const void * table, const int * ids, void * out, int T, int d, int n_vocab, void * stream);
JIB_EXPORT int jib_rmsnorm(const void * x, const void * residual, const float * w, void * out_norm, void * out_sum, int T, int d,
                           long long x_stride, float eps, void * stream);
// q_out: where the rotated RoPE part of token 0, head 0 goes; token t, head h at q_out + t * qo_row + h * qo_head (elements):
// into the absorbed-query buffer [T][H][r + dr] at offset r, or in place into q at offset dn.  ckv NULL: queries only (the
// layer reads another layer's latent rows).  rot_half: pairs (i, i + dr/2) instead of (2i, 2i + 1).  f32: fp32 activations and cache.
JIB_EXPORT int jib_mla_qkv_post(const void * q, long long q_stride, const void * ckv, long long ckv_stride, const float * kv_norm_w,
                                float eps, const float * rope_table, const int * positions, const int * slot_mapping, void * cache,
                                void * q_out, long long qo_row, long long qo_head, int T, int H, int dn, int dr, int r, int max_pos,
                                long long n_slots, int rot_half, int f32, int * status, void * stream);
JIB_EXPORT int jib_argmax(const float * logits, int * out, int n, int V, void * stream);
JIB_EXPORT int jib_topk(const float * logits, float * vals, int * ids, int n, int V, int k, void * stream);
JIB_EXPORT int jib_kv_block_copy(void * cache, long long layer_stride_elems, int n_layers, const int * src, const int * dst, int n,
                                 int block_elems, void * stream);
JIB_EXPORT int jib_gather_rows(const void * x, const int * src_row, void * out, int rows, int d, int n_src, void * stream);

// ---- MoE routing (moe.cu) ---------------------------------------------------------------------
// logits: fp32 scratch [T][E] (router outputs, kept for inspection).  ids / wts have k + n_shared columns: the last
// n_shared columns name the shared experts (ids E, E+1, ...; weight 1) so that they run in the grouped GEMMs.
// bias: added to the scores for the choice only (DeepSeek-V3); logit_bias: added to the router logits before anything else.
// g NULL: logits already holds the router outputs (fp32 activations).
// shared_gate: w_router and logits have a row / column more, E, and the shared experts' weight is sigmoid(logits[t][E]) instead of 1.
JIB_EXPORT int jib_moe_gate(const void * g, const float * w_router, const float * bias, const float * logit_bias, float * logits, int * ids,
                            float * wts, int T, int d, int E, int k, int n_group, int topk_group, float scale, int norm, int sigmoid,
                            int n_shared, int group_top2, int shared_gate, void * stream);
// jib_moe_gate + jib_moe_permute (over the k + n_shared id columns) in one launch, for T <= 64.  counter: one device int that is
// zero between launches.  norm_w != NULL: the rows of g are RMS-normalised first (as jib_rmsnorm would) and stored to g_out.
JIB_EXPORT int jib_moe_route_fused(const void * g, const float * w_router, const float * bias, float * logits, int * ids, float * wts,
                                   int * seg, int * src_token, int * dest, int * counter, int T, int d, int E, int k, int n_group,
                                   int topk_group, float scale, int norm, int sigmoid, int n_shared, int group_top2, int expert_base,
                                   int E_local, const float * norm_w, float eps, void * g_out, void * stream);
// Stable counting sort of the (token, k) pairs by local expert. dest[t*k+j] = sorted row or -1 (not local).
// seg has room for 2 * E_local + 1 ints: the E_local + 1 segment offsets, then the list of the experts that have rows (in
// order, -1 after the last): what jib_gemm_desc.expert_list takes.  (jib_moe_route_fused writes the same; the multi-CTA
// sort for large batches writes the offsets only.)  wts NULL, or [T][k]: row_wts[row] receives the weight of the pair in sorted row `row`.
JIB_EXPORT int jib_moe_permute(const int * ids, int T, int k, int expert_base, int E_local, int * seg, int * src_token, int * dest,
                               const float * wts, float * row_wts, void * stream);
// (expert, token tile) work list of a grouped launch with token-tile width bn: out[i] = tile << 16 | expert for every tile of
// every expert that has rows, in expert order, -1 up to cap.  cap >= rows / bn + E_local always suffices.
JIB_EXPORT int jib_moe_tile_list(const int * seg, int E_local, int bn, int * out, int cap, void * stream);
JIB_EXPORT int jib_moe_permute_multi(const int * ids, int T, int k, int expert_base, int E_local, int * seg, int * src_token, int * dest,
                                     int * tmp, const float * wts, float * row_wts, void * stream);
JIB_EXPORT int jib_moe_combine(const void * y, const int * dest, const float * wts, const void * shared, const void * residual,
                               void * out, int T, int k, int d, void * stream);
// The same followed by RMSNorm(out) * norm_w (fp32 weights, as jib_rmsnorm) in one launch; bitwise the two-launch results.
JIB_EXPORT int jib_moe_combine_norm(const void * y, const int * dest, const float * wts, const void * shared, const void * residual,
                                    const float * norm_w, void * out, void * out_norm, int T, int k, int d, float eps, void * stream);

// ---- attention (mla_attention.cu) -------------------------------------------------------------
// Split-KV absorbed MLA over the paged latent cache. q [T][H][r+dr], o_lat [T][H][r], cache rows: bf16, or fp32 with f32.
// window > 0: position i sees j with 0 <= i - j < window.  r <= 1024.
// part_o [T][n_splits][H][r] fp32 and part_ml [T][n_splits][H][2] fp32 are scratch.
JIB_EXPORT int jib_mla_attention(const void * q, const void * cache, const int * block_tables, int max_blocks, const int * seq_lens,
                                 const int * q_start, int n_seqs, int T, int H, int r, int dr, int block_size, float scale,
                                 int window, int n_splits, int f32, float * part_o, float * part_ml, void * o_lat, void * stream);

JIB_EXPORT int jib_mla_combine(const float * part_o, const float * part_ml, int n_splits, int T, int H, int r, void * o_lat,
                               void * stream);
// tcgen05 flash MLA (mla_flash_tcgen05.cu): r = 512, dr = 64, block size 64 only; qt = query tokens per CTA (1 or 2).
JIB_EXPORT int jib_mla_flash(const void * q, const void * cache, long long n_slots, const int * block_tables, int max_blocks,
                             const int * seq_lens, const int * q_start, int n_seqs, int T, int H, float scale, int window, int n_splits, int qt,
                             float * part_o, float * part_ml, void * o_lat, int * status, void * stream);

// ---- prefill attention in the per-head form (mha_prefill_tcgen05.cu): head dims 128 + 64 (keys), 128 (values) ---------------
// jib_kv_gather: lat [total_cap][row_elems] <- the cached latent rows of every sequence, in sequence order; kv_start [n_seqs].  pool null, or pooled
// rows (jib_gqa): those the sequence's last position sees come ahead of its own.
JIB_EXPORT int jib_kv_gather(const void * cache, long long n_slots, const int * block_tables, int max_blocks, const int * seq_lens,
                             int n_seqs, int block_size, int row_elems, const int * q_start, int window, int chunk, const void * pool, int pool_size,
                             int pool_rows, void * lat, int * kv_start, int total_cap, void * stream);
// q [T][H][192] (RoPE applied), kv [total][H][256] = k_nope | v, kpe [total][64] (row stride kpe_stride), out [T][H * 128].
JIB_EXPORT int jib_mha_prefill(const void * q, long long q_stride, const void * kv, const void * kpe, long long kpe_stride, long long total,
                               const int * q_start, const int * seq_lens, const int * kv_start, int n_seqs, int T, int H, float scale,
                               int window, int n_q_tiles, void * out, long long ldo, int * status, void * stream);

// ---- parallel blocks over an fp32 residual (parallel_block.cu), per-sequence state (recurrent.cu) ---------------------------
// What happens to a token's row once its residual value is known: x_out [T][d] fp32; with norm_w, h_out = row / rms * norm_w (with
// norm2_w too, h2_out = row / rms * norm2_w); with h_out but no norm_w, h_out = the row itself in the activation type; with
// conv_w ([taps][d] fp32, one token per sequence only), hc_out = h + causal convolution of h, whose last taps - 1 inputs live in
// conv_state [n_state][taps - 1][d] at row seq_slots[t] (negative: none) and are advanced.  positions[t] == 0 starts from zeros.
typedef struct jib_row_tail {
    void * x_out;
    const float * norm_w;
    void * h_out;
    const float * conv_w;
    void * hc_out;
    void * conv_state;
    const int * seq_slots;
    const int * positions;
    int * status;
    float eps;
    int taps, n_state;
    const float * norm2_w;     // null, or a second norm of the same row (not with conv_w)
    void * h2_out;
    int groups;                // > 1: the norms are taken over that many equal parts of the row, each by itself (embed_norm, scaled_update)
} jib_row_tail;
// x_out = scale * table[ids[t]], RMS-normed and times w unless w is null.
JIB_EXPORT int jib_embed_norm(const void * table, const int * ids, const float * w, float eps, float scale, int T, int d, int n_vocab, int f32,
                              const jib_row_tail * tail, void * stream);
// x_out = x + y / rms(y) * w (y [T][d] in the activation type); x_out may be x.
JIB_EXPORT int jib_post_norm(const float * x, const void * y, const float * w, float eps, int T, int d, int f32, const jib_row_tail * tail,
                             void * stream);
// x_out = x + mult * (sigmoid(gates[:, :d] + b1) * o + sigmoid(gates[:, d:2d] + b2) * sum_j wts[t][j] * y[dest[t][j]]); y NULL: no second
// sublayer.  x_out may be x.
JIB_EXPORT int jib_block_update(const float * x, float mult, const void * o, const void * gates, long long gate_stride, const float * b1,
                                const float * b2, const void * y, const int * dest, const float * wts, int k, int T, int d, int f32,
                                const jib_row_tail * tail, void * stream);
// x_out = x + s1 * o + s2 * (sum_j wts[t][j] * y[dest[t][j]] + g * f), s1, s2 [d]; any of o, y, f may be null (absent).  f [T][d]: a dense
// sublayer; g = sigmoid(f_gate[t * ld_gate]), 1 with f_gate null; s1, s2 or wts null: ones.  x_out may be x, or null: only the tail's norms.
JIB_EXPORT int jib_scaled_update(const float * x, const void * o, const float * s1, const void * y, const int * dest, const float * wts, int k,
                                 const void * f, const float * f_gate, long long ld_gate, const float * s2, int T, int d, int f32,
                                 const jib_row_tail * tail, void * stream);
JIB_EXPORT int jib_rms_rows(const float * x, const int * rows, const float * w, float eps, int n, int d, int n_src, int groups, int f32, void * out,
                            void * stream);
// out = h + causal convolution over time of h (w [taps][d] fp32), or with silu != 0 out = silu(bias + convolution); h [T][ldh], out
// [T][d]; sequence b continues from, and advances, its stored rows (state [n_state][taps - 1][d]).
JIB_EXPORT int jib_causal_conv(const void * h, long long ldh, const float * w, const float * bias, int silu, int taps, void * state, int n_state,
                               const int * seq_slots, const int * positions, const int * q_start, int n_seqs, int T, int d, int f32, void * out,
                               int * status, void * stream);
// Gated recurrence over zxg [T][>= 3W]; state [n_state][W] fp32; single: one token per sequence (row t = sequence t).
JIB_EXPORT int jib_mingru(const void * zxg, long long ld, const float * zb, const float * xb, float * state, int n_state,
                          const int * seq_slots, const int * positions, const int * q_start, int n_seqs, int T, int W, int single, int f32,
                          void * y, int * status, void * stream);

// ---- grouped-query attention over paged key / value rows (gqa_attention.cu) ------------------------------------------------
typedef struct jib_gqa {
    void * cache;              // [n_slots][row]: G * D key columns, then G * V value columns (activation type)
    const int * block_tables;  // [n_seqs][max_blocks]
    const int * seq_lens, * q_start, * positions;
    int * status;
    long long n_slots, row;
    int H, G, D, V, rot, block_size, max_blocks, n_seqs, T, max_pos;
    int window, chunk;         // position i sees j <= i with i - j < window (0: no window) and j / chunk == i / chunk (0: no chunks)
    int sink;                  // 1: the softmax' denominator also holds exp(0), or exp(sink_w[h])
    float scale, softcap;      // softcap 0: none
    float eps, out_scale;
    const float * sink_w;      // [H] or null
    // pool_size > 0 (with a window): position i also sees one key and value per block b of pool_size positions with
    // (b + 1) pool_size - 1 <= i - window, the mean of the block's cached rows.  It lies in row b - first of the pool_rows rows that go with the
    // cache block of the pooled block's last position, first = the first pooled block that ends there.
    void * pool;               // [blocks][pool_rows][row]
    const void * v_first;      // mix_v: values [T][ld_first]; cached are (1 - v_mix) v + v_mix v_first
    long long ld_first;
    int pool_size, pool_rows;
    int neighbours;            // rotated pairs are (2 i, 2 i + 1) instead of (i, i + rot / 2)
    int unit;                  // q and k over their root mean square, after the rotation
    int gate_each;             // the gate has a column per head and value channel instead of one per head
    int mix_v;
    float v_mix;
} jib_gqa;
// q, k, v: columns of the projection (row stride ld); q_norm, k_norm [D], or null: no norm.  rope [max_pos][rot / 2] pairs (cos, sin).  With a pool
// the pooled rows that are complete are stored as well; single: one token per sequence.
JIB_EXPORT int jib_gqa_qkv_post(const jib_gqa * m, const void * q, const void * k, const void * v, long long ld, const float * q_norm,
                                const float * k_norm, const float * rope, const int * slot_mapping, void * q_out, int single, int f32, void * stream);
// q [T][H][D]; gate null or [T][ld_gate] pre-activations of sigmoids; out [T][ldo].  single: one token per sequence.
// splits (<= 8): CTAs that share a row's keys.
JIB_EXPORT int jib_gqa_attention(const jib_gqa * m, const void * q, const void * gate, long long ld_gate, void * out, long long ldo, int single,
                                 int splits, int f32, void * stream);

// The same for prompt chunks on tcgen05 tensor cores (mha_prefill_tcgen05.cu): bf16, D = V = 128.  kv [total][row]: the rows jib_kv_gather
// copied; kv_start [n_seqs] the first of each sequence; n_q_tiles >= sum_b ceil(q_len_b / 128).
JIB_EXPORT int jib_gqa_prefill(const jib_gqa * m, const void * q, const void * kv, long long total, const int * kv_start, const void * gate,
                               long long ld_gate, int n_q_tiles, void * out, long long ldo, void * stream);

// ---- mixers with a matrix state per head (state_mix.cu) ----------------------------------------------------------------------
enum { JIB_STATE_DELTA = 0, JIB_STATE_LINEAR = 1, JIB_STATE_SSD = 2, JIB_STATE_HGRN = 3, JIB_STATE_MLSTM = 4 };
typedef struct jib_state_mix {
    // activations (bf16 or fp32): proj [T][ld] holds q (H / rep heads x K), k, v (H x V) and the pre-activation of the per-head
    // factor (s_off; H columns; DELTA, SSD) at these columns (HGRN has no k); dec_in [T][ld_dec] the decays' (H x K; not SSD), MLSTM: input |
    // forget gates' (2 H); gate [T][ld_gate] H x V (not HGRN)
    const void * proj, * dec_in, * gate;
    void * y;                  // [T][ldy] result, H x V columns
    // per-sequence state: [n_state][taps][n_conv] ring of convolution inputs (activation type), [n_state][H][K][V] fp32
    void * conv_state;
    float * state;
    const float * conv_w;      // [taps][n_conv]: columns conv0 .. conv0 + n_conv of proj are convolved (taps 0: none), last tap = current
    const float * conv_b;      // [n_conv] or null
    const float * bias;        // decays' (H x K), SSD's factor's (H), MLSTM's gates' (2 H)
    const float * neg_a;       // [H], not LINEAR
    const float * skip;        // [H], SSD
    const float * norm_w;      // [V], SSD, MLSTM [H x V]
    const int * seq_slots, * positions, * q_start;
    int * status;
    float * qk, * v, * dec, * s, * o;      // scratch: [T][2][H / rep][K], [T][H][V], [T][H][K] (SSD, MLSTM [T][H]), [T][H], [T][H][V]; MLSTM: V
                                           // rounded up to the next multiple of 4 above it
    void * chunk;              // null, or chunk_bytes >= jib_state_chunk_bytes: portions of bf16 go through the tensor cores (then qk, dec unused)
    long long ld, ld_dec, ld_gate, ldy, chunk_bytes;
    int kind, H, K, V, rep, taps, conv0, n_conv, q_off, k_off, v_off, s_off, norm_groups, n_state, n_seqs, T;
    float q_scale, inv_tau, eps, out_scale;
    const float * lower;       // [H x K], HGRN: lower bounds of the decays
    float * extra;             // [n_state][H][K + 1], MLSTM: what the keys add up to, then the running maximum of the gates
    float * tops;              // scratch [T][H], MLSTM: the running maximum at every token
    float gate_cap;            // MLSTM
} jib_state_mix;
// single: one token per sequence (row t = sequence t; scratch only for SSD: o).  K <= 512.
JIB_EXPORT int jib_state_mix_run(const jib_state_mix * m, int single, int f32, void * stream);
JIB_EXPORT long long jib_state_chunk_bytes(const jib_state_mix * m);

// ---- selective scan: a diagonal state per channel (selective_scan.cu) -------------------------------------------------------------
//   S[c][n] <- exp(dt_c a[c][n]) S[c][n] + dt_c x_c B_n;   y_c = (sum_n S[c][n] C_n + skip_c x_c) * silu(z_c) * out_scale,   dt = softplus(dt_c + bias_c)
// over ch channels (a multiple of 8) with N states each (a multiple of 8, at most 256).
typedef struct jib_scan {
    const void * x, * z, * bc, * dt;       // activations: [T][ldx], [T][ldz], [T][ldbc] = B | C, [T][lddt]
    void * y;                  // [T][ldy]
    const float * neg_a;       // [ch][N]
    const float * skip, * dt_bias;         // [ch]
    float * state;             // [n_state][ch][N]
    const int * seq_slots, * positions, * q_start;
    int * status;
    long long ldx, ldz, ldbc, lddt, ldy;
    int ch, N, n_state, n_seqs, T;
    float out_scale;
} jib_scan;
// single: one token per sequence (row t = sequence t).
JIB_EXPORT int jib_selective_scan(const jib_scan * m, int single, int f32, void * stream);

// ---- expert-parallel all-to-all over peer memory (ep_alltoall.cu); ctx is a JibEpCtx (ep_alltoall.h) ---------
JIB_EXPORT int jib_ep_plan(const int * ids, int T, int k, const struct JibEpCtx * ctx, int site, int * seg, int * pair_dst, void * stream);
JIB_EXPORT int jib_ep_push(const void * x, const int * pair_dst, int T, int k, const struct JibEpCtx * ctx, int site, const int * seg,
                           int * done_counter, void * row_ptr, void * stream);
JIB_EXPORT int jib_ep_combine(const float * wts, const int * pair_dst, const void * shared, const void * residual, void * out, int T,
                              int k, const struct JibEpCtx * ctx, int site, void * stream);

#ifdef __cplusplus
}
#endif
