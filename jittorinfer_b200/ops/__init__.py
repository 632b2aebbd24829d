"""Op front-end used by the model graph.

CUDA tensors go to the hand-written sm_100a kernels (``ops.native``, loaded from the in-tree
``libjib200_kernels.so``); if that library is missing on a GPU machine the import fails loudly —
there is no silent fallback.  CPU tensors (tests, host tools) use ``ops.reference``.
``JITTORINFER_OPS=torch`` selects the PyTorch/cuBLAS implementation on the GPU as well: that is
the measured baseline, never the default.
"""
from __future__ import annotations

import os

import torch

from . import reference as ref

_FORCE_TORCH = os.environ.get("JITTORINFER_OPS", "").lower() == "torch"
_native = None


def nat():
    """The ctypes binding module; raises if the CUDA library is not built."""
    global _native
    if _native is None:
        from . import native as _n
        _n.load()
        _native = _n
    return _native


def use_native(t: torch.Tensor) -> bool:
    return t.is_cuda and not _FORCE_TORCH


def set_force_torch(flag: bool) -> None:
    global _FORCE_TORCH
    _FORCE_TORCH = bool(flag)


def force_torch() -> bool:
    return _FORCE_TORCH


def embed_gather(table, ids):
    return nat().embed_gather(table, ids) if use_native(table) else ref.embed_gather(table, ids)


def select_rows(x, rows):
    """x[rows] (the reference's inp_out_ids row selection, src/llama-graph-deepseek2.cpp:302-308)."""
    if use_native(x) and x.dtype == torch.bfloat16:
        return nat().gather_rows(x, rows)
    return x[rows.long()].contiguous()


def rmsnorm(x, w, eps, residual=None):
    return nat().rmsnorm(x, w, eps, residual) if use_native(x) else ref.rmsnorm(x, w, eps, residual)


def linear(x, w, residual=None, out_dtype=None, unary=None):
    """f(x w^T) + residual (a bias: one row expanded over the tokens); ``unary``: None, ("relu2",), ("gelu",) or ("cap", scale, softcap)."""
    if use_native(x) and x.dtype == torch.bfloat16:
        return nat().linear(x, w, residual, out_dtype, unary)
    return ref.linear(x, w, residual, out_dtype, unary)


def gateup_silu(x, wg, wu):
    if use_native(x) and x.dtype == torch.bfloat16:
        return nat().gateup_silu(x, wg, wu)
    return ref.gateup_silu(x, wg, wu)


def gateup(x, wg, wu, act):
    """act(x wg^T) * (x wu^T), ``act`` "silu" or "gelu_tanh"; fp32 operands take the library's products."""
    if use_native(x) and x.dtype == torch.bfloat16:
        return nat().gateup(x, wg, wu, act)
    return ref.gateup(x, wg, wu, act)


def mla_qkv_post(q, ckv, kv_norm_w, eps, rope_table, positions, slot_mapping, cache, q_out, n_head, dn, dr, r, rot_half=False):
    f = nat().mla_qkv_post if use_native(q) else ref.mla_qkv_post
    return f(q, ckv, kv_norm_w, eps, rope_table, positions, slot_mapping, cache, q_out, n_head, dn, dr, r, rot_half)


def q_absorb(q_nope, w_uk, q_out, r):
    return (nat().q_absorb if use_native(q_nope) else ref.q_absorb)(q_nope, w_uk, q_out, r)


def v_up(o_lat, w_uv):
    return (nat().v_up if use_native(o_lat) else ref.v_up)(o_lat, w_uv)


def mla_attention(q, cache, block_tables, seq_lens, q_start, scale, r, block_size, max_q_len=None, meta=None, window=0):
    if use_native(q):
        return nat().mla_attention(q, cache, block_tables, seq_lens, q_start, scale, r, block_size, max_q_len, meta, window)
    return ref.mla_attention(q, cache, block_tables, seq_lens, q_start, scale, r, block_size, window)


def moe_gate(g, w_router, bias, k, n_group, topk_group, scale, norm, sigmoid, n_shared=0, group_top2=False, route=None, pre_norm=None,
             logit_bias=None, shared_gate=False):
    """``w_router`` fp32, or bf16 with bf16 activations (products of exact operands on the tensor cores, fp32 sums).  ``shared_gate``: the last row of ``w_router`` is the shared experts' gate, not an expert: their weight is its sigmoid (``n_shared``
    columns), and the router outputs' last column is returned as well.
    ``route=(expert_base, E_local)`` tells the CUDA path which local expert sort follows (see ``native.moe_gate``).
    ``pre_norm=(weight, eps)``: ``g`` is the un-normalised block input; returns (ids, wts, rmsnorm(g) * weight) -- on the CUDA
    path the router launch of a decode batch normalises the rows itself."""
    if use_native(g):
        return nat().moe_gate(g, w_router, bias, k, n_group, topk_group, scale, norm, sigmoid, n_shared, group_top2, route, pre_norm,
                              logit_bias, shared_gate)
    if pre_norm is not None:
        g, _ = ref.rmsnorm(g, pre_norm[0], pre_norm[1])
        return ref.moe_gate(g, w_router, bias, k, n_group, topk_group, scale, norm, sigmoid, n_shared, group_top2) + (g,)
    return ref.moe_gate(g, w_router, bias, k, n_group, topk_group, scale, norm, sigmoid, n_shared, group_top2, logit_bias, shared_gate)


def moe_routed(x, ids, wts, wg, wu, wd):
    """(expert outputs of the (token, choice) pairs, row of each pair); the weighted sum is the caller's (``block_update``).  ``wg`` None: experts
    without a gate, gelu(w x up^T) down^T -- the weight multiplies their input, the sum of the outputs is the result."""
    return (nat() if use_native(x) else ref).moe_routed(x, ids, wts, wg, wu, wd)


def moe_experts(x, ids, wts, wg, wu, wd, expert_base=0):
    if use_native(x) and x.dtype == torch.bfloat16:
        return nat().moe_experts(x, ids, wts, wg, wu, wd, expert_base)
    return ref.moe_experts(x, ids, wts, wg, wu, wd, expert_base)


def moe_ffn(x, residual, ids, wts, wg, wu, wd, wgs, wus, wds, expert_base=0, n_expert=None, norm=None):
    """``n_expert``: size of the router's expert set (lets the CUDA path estimate how many local experts a batch hits).
    ``norm=(weight, eps)``: returns (out, rmsnorm(out) * weight) -- the CUDA path computes both in the combine launch."""
    if use_native(x) and x.dtype == torch.bfloat16:
        return nat().moe_ffn(x, residual, ids, wts, wg, wu, wd, wgs, wus, wds, expert_base, n_expert, norm)
    out = ref.moe_ffn(x, residual, ids, wts, wg, wu, wd, wgs, wus, wds, expert_base)
    return (out, ref.rmsnorm(out, norm[0], norm[1])[0]) if norm is not None else out


def fused_combine_norm() -> bool:
    """Whether the model should ask ``moe_ffn`` for the next block's norm as well (one launch on the CUDA path;
    JIB_FUSED_COMBINE_NORM=0 keeps the two launches for A/B measurements)."""
    return os.environ.get("JIB_FUSED_COMBINE_NORM", "1") == "1"


# ---- parallel blocks over an fp32 residual stream, per-sequence state -------------------------------------------------------------
# ``nxt`` = (norm weight, eps, conv): the norm the next block reads, computed in the same pass; conv = None, or -- one token per
# sequence only -- (weights [taps, d], state, seq_slots, positions) of that block's input convolution.  Or a ``specs.RowNorms``: one or
# two norms of the row, or the row in the activation type; the second comes back in the place of h + convolution.
def embed_norm(table, ids, w, eps, nxt=None, scale=1.0):
    """(x fp32 = norm of the scaled embedding rows (``w`` None: the rows themselves), h, h + convolution)."""
    return (nat() if use_native(table) else ref).embed_norm(table, ids, w, eps, nxt, scale)


def post_norm(x, y, w, eps, nxt=None):
    """(x + norm(y) * w, h) with ``nxt`` = (norm weight, eps, None) of the sublayer that follows; x may be overwritten."""
    return (nat() if use_native(x) else ref).post_norm(x, y, w, eps, nxt)


def block_update(x, mult, o, gates, b1, b2, moe=None, nxt=None):
    """(x + mult * (sigmoid(g1 + b1) * o + sigmoid(g2 + b2) * combine(moe)), h, h + convolution); x may be overwritten."""
    return (nat() if use_native(x) else ref).block_update(x, mult, o, gates, b1, b2, moe, nxt)


def scaled_update(x, o, s1, s2=None, moe=None, dense=None, dense_gate=None, nxt=None, dtype=None):
    """(x + s1 * o + s2 * (combine(moe) + sigmoid(dense_gate) * dense), h, h2); ``o``, ``moe`` = (rows, row of each pair, weights) and
    ``dense`` may be None, ``s1``, ``s2``, the weights or ``dense_gate`` [T] None is a factor of one; ``dtype``: activation type (default: that of the sublayers' rows); x may be
    overwritten."""
    return (nat() if use_native(x) else ref).scaled_update(x, o, s1, s2, moe, dense, dense_gate, nxt, dtype)


def rms_rows(x, rows, w, eps, dtype, groups=1):
    return (nat() if use_native(x) else ref).rms_rows(x, rows, w, eps, dtype, groups)


def causal_conv(h, w, state, seq_slots, positions, q_start, bias=None):
    """h + convolution, or with ``bias`` silu(convolution + bias); h may be a slice of columns."""
    return (nat() if use_native(h) else ref).causal_conv(h, w, state, seq_slots, positions, q_start, bias)


def mingru(zxg, zb, xb, state, seq_slots, positions, q_start, single=False):
    return (nat() if use_native(zxg) else ref).mingru(zxg, zb, xb, state, seq_slots, positions, q_start, single)


# ---- mixers described by a spec (ops/specs.py) ------------------------------------------------------------------------------------
def state_mix(m, proj, dec_in, gate, conv_state, state, seq_slots, positions, q_start, single, out, extra=None):
    """A mixer with a matrix state per head over a batch, convolution to gated norm; result columns go to ``out`` (a view).  ``state`` [n, heads,
    dim, vdim] fp32.  "mlstm": ``dec_in`` [T, 2 heads] = input | forget gates' pre-activations, ``extra`` [n, heads, dim + 1] fp32 = what the
    keys add up to, the running maximum."""
    return (nat() if use_native(proj) else ref).state_mix(m, proj, dec_in, gate, conv_state, state, seq_slots, positions, q_start, single, out, extra)


def selective_scan(m, x, z, bc, dt, state, seq_slots, positions, q_start, single, out):
    """``m``: ``specs.SelectiveScan``; ``bc`` = B | C, ``dt`` the step sizes' projection; result columns go to ``out`` (a view)."""
    return (nat() if use_native(x) else ref).selective_scan(m, x, z, bc, dt, state, seq_slots, positions, q_start, single, out)


def gqa_qkv_post(m, q, k, v, rope_table, positions, slot_mapping, cache, v_first=None, pooled=None):
    """``v_first``: the values that ``m.v_mix`` mixes in.  ``pooled`` (with ``m.pool``): (pooled rows, block tables, seq_lens, q_start, block size, one
    token per sequence); the means of the blocks that are now complete are stored as well."""
    return (nat() if use_native(q) else ref).gqa_qkv_post(m, q, k, v, rope_table, positions, slot_mapping, cache, v_first, pooled)


def gqa_attention(m, q, cache, gate, block_tables, seq_lens, q_start, block_size, max_q_len, meta, out, pool=None):
    """Result columns go to ``out`` (a view); ``pool``: the pooled rows of ``m.pool``."""
    return (nat() if use_native(q) else ref).gqa_attention(m, q, cache, gate, block_tables, seq_lens, q_start, block_size, max_q_len, meta, out, pool)


def argmax(logits):
    return nat().argmax(logits) if use_native(logits) else ref.argmax(logits)


def topk_logits(logits, k):
    return nat().topk_logits(logits, k) if use_native(logits) else ref.topk_logits(logits, k)


def sample_topk(vals, ids, params):
    """One id per row from sorted top-k candidates: top-k / top-p / min-p / temperature and one uniform per row."""
    return nat().sample_topk(vals, ids, params) if use_native(vals) else ref.sample_topk(vals, ids, params)


def kv_block_copy(cache, src_blocks, dst_blocks, block_size):
    f = nat().kv_block_copy if use_native(cache) else ref.kv_block_copy
    return f(cache, src_blocks, dst_blocks, block_size)
