"""Plain-PyTorch implementations of every op the model graph uses.

These are (a) the CPU path (tests, host-only tools), (b) the fp32 numerics reference the CUDA
kernels are tested against, and (c) on a GPU, the torch/cuBLAS *baseline* the native kernels are
measured against (``JITTORINFER_OPS=torch``).  Semantics follow the reference graph
(src/llama-graph-deepseek2.cpp:113-405); each function names the reference op it stands for.
"""
from __future__ import annotations

import math
from typing import Optional, Tuple

import torch
import torch.nn.functional as F

from .specs import RowNorms


def embed_gather(table: torch.Tensor, ids: torch.Tensor) -> torch.Tensor:
    """ggml get_rows on the token embedding (src/llama-graph-utils.cpp:7-40)."""
    return table[ids.long()]


def rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float, residual: Optional[torch.Tensor] = None
            ) -> Tuple[torch.Tensor, torch.Tensor]:
    """(normed, summed): summed = x + residual (or x); normed = rmsnorm(summed) * w in fp32 statistics."""
    s = x if residual is None else (x.float() + residual.float()).to(x.dtype)
    sf = s.float()
    n = sf * torch.rsqrt(sf.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    return n.to(x.dtype), s


def unary_of(y: torch.Tensor, unary) -> torch.Tensor:
    """None, ("relu2",): max(y, 0)^2, ("gelu",): the exact gelu, or ("cap", s, c): c tanh(s y / c), s y with c = 0."""
    if unary is None:
        return y
    if unary[0] == "gelu":
        return F.gelu(y.float())
    if unary[0] == "relu2":
        return torch.relu(y).square()
    y = y.float() * unary[1]
    return unary[2] * torch.tanh(y / unary[2]) if unary[2] else y


def linear(x: torch.Tensor, w: torch.Tensor, residual: Optional[torch.Tensor] = None,
           out_dtype: Optional[torch.dtype] = None, unary=None) -> torch.Tensor:
    """y = f(x @ w.T) (+ residual); fp32 accumulate."""
    if x.dtype == torch.float32 or x.is_cuda:
        y = x @ w.T if out_dtype in (None, x.dtype) else (x.float() @ w.float().T)
    else:
        y = (x.float() @ w.float().T)
    y = unary_of(y, unary)
    if residual is not None:
        y = y.float() + residual.float()
    return y.to(out_dtype or x.dtype)


def gateup_silu(x: torch.Tensor, wg: torch.Tensor, wu: torch.Tensor) -> torch.Tensor:
    """silu(x wg^T) * (x wu^T) (src/llama-graph-ffn.cpp:4-126, LLM_FFN_SILU + LLM_FFN_PAR)."""
    g = linear(x, wg, out_dtype=torch.float32)
    u = linear(x, wu, out_dtype=torch.float32)
    return (F.silu(g) * u).to(x.dtype)


def gateup(x: torch.Tensor, wg: torch.Tensor, wu: torch.Tensor, act: str) -> torch.Tensor:
    """act(x wg^T) * (x wu^T), ``act`` "silu" or "gelu_tanh"."""
    g = linear(x, wg, out_dtype=torch.float32)
    u = linear(x, wu, out_dtype=torch.float32)
    return ((F.silu(g) if act == "silu" else F.gelu(g, approximate="tanh")) * u).to(x.dtype)


def yarn_table(n_pos: int, dr: int, freq_base: float, freq_scale: float, ext_factor: float, attn_factor: float,
               corr_lo: float, corr_hi: float, device="cpu") -> torch.Tensor:
    """[n_pos, dr/2, 2] fp32 (cos, sin) incl. magnitude factor — the GE path's RopeCache
    (ggml/src/ggml-cann/rope_cache.cpp:16-79) restated; formula ggml-cpu.c:10272-10305."""
    i = torch.arange(dr // 2, dtype=torch.float64)
    pos = torch.arange(n_pos, dtype=torch.float64)
    te = pos[:, None] * freq_base ** (-2.0 * i / dr)[None, :]
    ti = freq_scale * te
    if ext_factor != 0.0:
        ramp = 1.0 - torch.clamp((i - corr_lo) / max(0.001, corr_hi - corr_lo), 0.0, 1.0)
        mix = ramp * ext_factor
        theta = ti * (1.0 - mix) + te * mix
        m = attn_factor * (1.0 + 0.1 * math.log(1.0 / freq_scale))
    else:
        theta, m = ti, attn_factor
    return torch.stack([torch.cos(theta) * m, torch.sin(theta) * m], dim=-1).float().to(device)


def _rope(x: torch.Tensor, cs: torch.Tensor, half: bool = False) -> torch.Tensor:
    """x [T, ..., dr]; cs [T, dr/2, 2].  Pairs are neighbours (2i, 2i + 1), or with ``half`` (i, i + dr/2)."""
    shp = x.shape
    c, s = cs[..., 0], cs[..., 1]
    while c.dim() < x.dim():
        c, s = c.unsqueeze(1), s.unsqueeze(1)
    if half:
        x0, x1 = x.float().chunk(2, dim=-1)
        return torch.cat([x0 * c - x1 * s, x0 * s + x1 * c], dim=-1)
    xp = x.float().reshape(*shp[:-1], shp[-1] // 2, 2)
    x0, x1 = xp[..., 0], xp[..., 1]
    return torch.stack([x0 * c - x1 * s, x0 * s + x1 * c], dim=-1).reshape(shp)


def mla_qkv_post(q: torch.Tensor, ckv: torch.Tensor, kv_norm_w: torch.Tensor, eps: float, rope_table: torch.Tensor,
                 positions: torch.Tensor, slot_mapping: torch.Tensor, cache: torch.Tensor,
                 q_out: torch.Tensor, n_head: int, dn: int, dr: int, r: int, rot_half: bool = False) -> torch.Tensor:
    """RMSNorm(c) + RoPE(k_pe) + latent-cache write + RoPE(q_pe)  (src/llama-graph-deepseek2.cpp:197-240).

    q [T, H*(dn+dr)], ckv [T, r+dr]; cache [n_slots, r+dr]; q_out [T, H, r+dr]: only the rope tail
    ``q_out[..., r:]`` is written here (the nope part is absorbed by :func:`q_absorb`).
    Rows with ``slot_mapping < 0`` are padding and are skipped.  ``ckv`` None: another layer has written the rows, only the
    queries are rotated.  Returns q_nope [T,H,dn] (a view).
    """
    T = q.shape[0]
    cs = rope_table[positions.long()]
    if ckv is not None:
        c = ckv[:, :r].float()
        c = c * torch.rsqrt(c.pow(2).mean(-1, keepdim=True) + eps) * kv_norm_w.float()
        kpe = _rope(ckv[:, r:], cs, rot_half)
        row = torch.cat([c, kpe], dim=-1).to(cache.dtype)
        valid = slot_mapping >= 0
        cache[slot_mapping[valid].long()] = row[valid]
    qv = q.reshape(T, n_head, dn + dr)
    q_out[..., r:] = _rope(qv[..., dn:], cs, rot_half).to(q_out.dtype)
    return qv[..., :dn]


def q_absorb(q_nope: torch.Tensor, w_uk: torch.Tensor, q_out: torch.Tensor, r: int) -> None:
    """q_out[..., :r] = q_nope[T,H,dn] @ w_uk[H,r,dn]^T  (src/llama-graph-attn.cpp:269-275)."""
    q_out[..., :r] = torch.einsum("thd,hrd->thr", q_nope.float(), w_uk.float()).to(q_out.dtype)


def v_up(o_lat: torch.Tensor, w_uv: torch.Tensor) -> torch.Tensor:
    """o[T, H*dv] = o_lat[T,H,r] @ w_uv[H,dv,r]^T  (src/llama-graph-attn.cpp:316-317)."""
    o = torch.einsum("thr,hvr->thv", o_lat.float(), w_uv.float())
    return o.reshape(o.shape[0], -1).to(o_lat.dtype)


def mla_attention(q: torch.Tensor, cache: torch.Tensor, block_tables: torch.Tensor, seq_lens: torch.Tensor,
                  q_start: torch.Tensor, scale: float, r: int, block_size: int, window: int = 0) -> torch.Tensor:
    """Weight-absorbed MLA over the paged latent cache (src/llama-graph-attn.cpp:219-342).

    q [T,H,r+dr]; cache [n_blocks*block_size, r+dr]; sequence b owns query rows
    q_start[b]:q_start[b+1] (its *last* tokens) and kv length seq_lens[b].  ``window`` > 0: position i sees j with
    0 <= i - j < window.  Returns o_lat [T,H,r].
    """
    T, H, _ = q.shape
    out = torch.zeros(T, H, r, dtype=q.dtype, device=q.device)
    qs = q_start.tolist()
    sl = seq_lens.tolist()
    for b in range(len(sl)):
        q0, q1, S = qs[b], qs[b + 1], sl[b]
        if q1 <= q0 or S <= 0:
            continue
        nb = (S + block_size - 1) // block_size
        blocks = block_tables[b, :nb].long()
        idx = (blocks[:, None] * block_size + torch.arange(block_size, device=q.device)[None, :]).reshape(-1)[:S]
        lat = cache[idx].float()                                   # [S, r+dr]
        qq = q[q0:q1].float()                                      # [Tq,H,r+dr]
        s = torch.einsum("thk,sk->hts", qq, lat) * scale
        Tq = q1 - q0
        pos = S - Tq + torch.arange(Tq, device=q.device)
        vis = torch.arange(S, device=q.device)[None, :] <= pos[:, None]
        if window > 0:
            vis &= torch.arange(S, device=q.device)[None, :] > pos[:, None] - window
        s = s.masked_fill(~vis[None], float("-inf"))
        p = torch.softmax(s, dim=-1)
        out[q0:q1] = torch.einsum("hts,sr->thr", p, lat[:, :r]).to(q.dtype)
    return out


def moe_gate(g: torch.Tensor, w_router: torch.Tensor, bias: Optional[torch.Tensor], k: int, n_group: int,
             topk_group: int, scale: float, norm: bool, sigmoid: bool, n_shared: int = 0,
             group_top2: bool = False, logit_bias: Optional[torch.Tensor] = None, shared_gate: bool = False):
    """Router matmul (fp32) + softmax/sigmoid + [group-limited] top-k + renorm/scale
    (src/llama-graph-ffn.cpp:145-197).  ``bias`` takes part in the choice only, ``logit_bias`` is part of the logits (with
    softmax and ``norm`` the weights are then a softmax over the chosen logits).  Returns ids [T,k] int32, weights [T,k] fp32; with
    ``shared_gate`` also the outputs of the router's last row, whose sigmoid is then the shared experts' weight."""
    logits = g.float() @ w_router.float().T
    gate = None
    if shared_gate:
        logits, gate = logits[:, :-1], logits[:, -1]
    if logit_bias is not None:
        logits = logits + logit_bias.float()
    probs = torch.sigmoid(logits) if sigmoid else torch.softmax(logits, dim=-1)
    sel = probs if bias is None else probs + bias.float()
    T, E = sel.shape
    if n_group > 1:
        grouped = sel.view(T, n_group, E // n_group)
        gs = grouped.topk(2, dim=-1).values.sum(-1) if group_top2 and E // n_group >= 2 else grouped.max(dim=-1).values
        order = torch.sort(gs, dim=-1, descending=True, stable=True).indices[:, :topk_group]
        mask = torch.zeros_like(gs, dtype=torch.bool).scatter_(1, order, True)
        sel = sel.masked_fill(~mask[:, :, None].expand(T, n_group, E // n_group).reshape(T, E), float("-inf"))
    ids = torch.sort(sel, dim=-1, descending=True, stable=True).indices[:, :k]
    w = torch.gather(probs, 1, ids)
    if norm:
        w = w / w.sum(-1, keepdim=True)
    ids, w = ids.int(), (w * scale).float()
    if n_shared:        # shared experts as always-selected experts E, E+1, ... with weight 1
        sh = torch.arange(E, E + n_shared, dtype=torch.int32, device=ids.device)[None].expand(T, n_shared)
        ids = torch.cat([ids, sh], dim=1)
        one = torch.ones(T, 1, dtype=w.dtype, device=w.device) if gate is None else torch.sigmoid(gate)[:, None]
        w = torch.cat([w, one.expand(T, n_shared)], dim=1)
    return (ids.contiguous(), w.contiguous()) + ((gate,) if shared_gate else ())


def moe_experts(x: torch.Tensor, ids: torch.Tensor, wts: torch.Tensor, wg: torch.Tensor, wu: torch.Tensor,
                wd: torch.Tensor, expert_base: int = 0) -> torch.Tensor:
    """sum_k w_k * down_e(silu(gate_e x) * up_e x) over the *local* experts
    [expert_base, expert_base + wg.shape[0]) (ggml_moe_fused with start/end expert,
    src/llama-graph-ffn.cpp:205-234).  Returns fp32 [T, d]."""
    T, d = x.shape
    E_local = wg.shape[0]
    out = torch.zeros(T, d, dtype=torch.float32, device=x.device)
    ids_l = ids.long() - expert_base
    for e in range(E_local):
        tok, slot = torch.nonzero(ids_l == e, as_tuple=True)
        if tok.numel() == 0:
            continue
        xe = x[tok]
        h = gateup_silu(xe, wg[e], wu[e])
        y = linear(h, wd[e], out_dtype=torch.float32)
        out.index_add_(0, tok, y * wts[tok, slot][:, None])
    return out


def moe_ffn(x, residual, ids, wts, wg, wu, wd, wgs, wus, wds, expert_base=0):
    """residual + shared_experts(x) + routed experts (src/llama-graph-deepseek2.cpp:343-362)."""
    out = moe_experts(x, ids, wts, wg, wu, wd, expert_base)
    if wgs is not None:
        out = out + linear(gateup_silu(x, wgs, wus), wds, out_dtype=torch.float32)
    if residual is not None:
        out = out + residual.float()
    return out.to(x.dtype)


def argmax(logits: torch.Tensor) -> torch.Tensor:
    return torch.argmax(logits.float(), dim=-1).int()


def topk_logits(logits: torch.Tensor, k: int) -> Tuple[torch.Tensor, torch.Tensor]:
    """Device "presample" (src/llama-execute-decode.cpp:132-154): top-k values fp32 + ids int32, sorted."""
    v, i = torch.topk(logits.float(), k, dim=-1, sorted=True)
    return v, i.int()


def sample_topk(vals: torch.Tensor, ids: torch.Tensor, params: torch.Tensor) -> torch.Tensor:
    """One token id per row from its top-k candidates, the device form of the chain top_k -> top_p -> min_p -> temperature
    -> dist (common/sampling_local.cpp:153-209).  ``vals`` / ``ids`` [n, k] sorted by value, descending; ``params`` [n, 5]
    fp32 = temperature (<= 0: best candidate), top_k (<= 0: all), top_p (>= 1: off), min_p (<= 0: off), u in [0, 1).
    Sorted candidates make every truncation a prefix: rank < top_k; probability mass before the candidate < top_p (softmax
    of the untempered logits of the top-k set); logit >= best + ln(min_p)."""
    v = vals.float()
    n, k = v.shape
    pr = params.float()
    temp, top_k, top_p, min_p, u = (pr[:, i:i + 1] for i in range(5))
    rank = torch.arange(k, device=v.device)[None]
    keep = (top_k <= 0) | (rank < top_k)
    m = v[:, :1]
    e = torch.exp(v - m) * keep
    before = (torch.cumsum(e, -1) - e) / e.sum(-1, keepdim=True)
    keep = keep & ((top_p >= 1.0) | (before < top_p))
    keep = keep & ((min_p <= 0) | (v >= m + torch.log(min_p.clamp_min(1e-30))))
    keep[:, 0] = True
    keep = torch.cumprod(keep.int(), -1).bool()                       # a prefix, as the sequential form breaks at the first miss
    w = torch.exp((v - m) / temp.clamp_min(1e-6)) * keep
    cdf = torch.cumsum(w, -1)
    pick = (cdf <= u * cdf[:, -1:]).sum(-1)
    last = keep.sum(-1) - 1
    pick = torch.minimum(pick, last)
    pick = torch.where(temp[:, 0] <= 0, torch.zeros_like(pick), pick)
    return ids.gather(1, pick[:, None].long())[:, 0].int()


def kv_block_copy(cache: torch.Tensor, src_blocks: torch.Tensor, dst_blocks: torch.Tensor, block_size: int) -> None:
    """Defrag move list (src/llama-graph-defrag.cpp:23-85) on paged blocks. cache [L, n_slots, row]."""
    L = cache.shape[0]
    c = cache.view(L, -1, block_size, cache.shape[-1])
    c[:, dst_blocks.long()] = c[:, src_blocks.long()]


def moe_routed(x, ids, wts, wg, wu, wd):
    """Expert outputs of every (token, choice) pair: (y [T*k, d], dest [T, k] row of each pair); here in pair order.  ``wg`` None: experts
    gelu(w x up^T) down^T, the weight on their input."""
    T, k = ids.shape
    y = torch.zeros(T * k, x.shape[1], dtype=x.dtype, device=x.device)
    flat = ids.reshape(-1).long()
    for e in range(wu.shape[0]):
        rows = torch.nonzero(flat == e).reshape(-1)
        if rows.numel() and wg is None:
            u = linear(x[rows // k], wu[e], out_dtype=torch.float32) * wts.reshape(-1)[rows][:, None]
            y[rows] = linear(F.gelu(u).to(x.dtype), wd[e])
        elif rows.numel():
            y[rows] = linear(gateup_silu(x[rows // k], wg[e], wu[e]), wd[e])
    return y, torch.arange(T * k, dtype=torch.int32, device=x.device).view(T, k)


# ---- blocks over an fp32 residual stream whose sublayers read one norm (csrc/kernels/parallel_block.cu) ------------------------
def _group_rms(x, groups, eps):
    v = x.reshape(x.shape[0], groups, -1)
    return (v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps)).reshape(x.shape)


def _finish_row(x, nxt, dtype):
    """x fp32 -> (x, h, hc) for ``nxt`` = (norm weight, eps, conv) with conv = None or (w [taps, d], state, seq_slots, positions), or a
    ``RowNorms``."""
    if nxt is None:
        return x, None, None
    if isinstance(nxt, RowNorms):
        if nxt.w1 is None:
            return x, x.to(dtype, copy=True), None
        n = _group_rms(x, nxt.groups, nxt.eps)
        return x, (n * nxt.w1).to(dtype), None if nxt.w2 is None else (n * nxt.w2).to(dtype)
    w, eps, conv = nxt
    h = (x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w).to(dtype)
    if conv is None:
        return x, h, None
    cw, state, slots, positions = conv
    n = torch.arange(x.shape[0] + 1, dtype=torch.int32)
    return x, h, causal_conv(h, cw, state, slots, positions, n)


def embed_norm(table, ids, w, eps, nxt=None, scale=1.0):
    v = table[ids.long()].float() * scale
    if w is None:
        return _finish_row(v, nxt, table.dtype)
    return _finish_row(v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps) * w, nxt, table.dtype)


def block_update(x, mult, o, gates, b1, b2, moe=None, nxt=None):
    """x + mult * (sigmoid(g1 + b1) * o + sigmoid(g2 + b2) * combine(moe)), ``moe`` = (y, dest, wts) or None."""
    d = x.shape[1]
    s = torch.sigmoid(gates[:, :d].float() + b1) * o.float()
    if moe is not None:
        y, dest, wts = moe
        f = (y.float()[dest.long()] * wts[..., None]).sum(1)
        s = s + torch.sigmoid(gates[:, d:2 * d].float() + b2) * f
    return _finish_row(x + mult * s, nxt, o.dtype)


def post_norm(x, y, w, eps, nxt=None):
    v = y.float()
    return _finish_row(x + v * torch.rsqrt(v.pow(2).mean(-1, keepdim=True) + eps) * w, nxt, y.dtype)[:2]


def scaled_update(x, o, s1, s2=None, moe=None, dense=None, dense_gate=None, nxt=None, dtype=None):
    """x + s1 * o + s2 * (combine(moe) + sigmoid(dense_gate) * dense), ``moe`` = (y, dest, wts); o, moe, dense may be None; s1, s2, wts None: one."""
    dtype = dtype or next((t.dtype for t in (o, dense, moe[0] if moe is not None else None) if t is not None), x.dtype)
    v = x
    if o is not None:
        v = v + (o.float() if s1 is None else s1 * o.float())
    f = None
    if moe is not None:
        y, dest, wts = moe
        f = y.float()[dest.long()]
        f = (f if wts is None else f * wts[..., None]).sum(1)
    if dense is not None:
        g = dense.float() if dense_gate is None else torch.sigmoid(dense_gate.float())[:, None] * dense.float()
        f = g if f is None else f + g
    return _finish_row(v if f is None else v + f if s2 is None else v + s2 * f, nxt, dtype)


def rms_rows(x, rows, w, eps, dtype, groups=1):
    return (_group_rms(x if rows is None else x[rows.long()], groups, eps) * w).to(dtype)


def causal_conv(h, w, state, seq_slots, positions, q_start, bias=None):
    """h + causal convolution over time, w [taps, d], or with ``bias`` silu(convolution + bias); ``state`` [n, taps - 1, d] holds each
    sequence's last inputs."""
    out = torch.empty(h.shape, dtype=h.dtype, device=h.device)
    taps = w.shape[0]
    qs = q_start.tolist()
    for b in range(len(qs) - 1):
        q0, q1 = qs[b], qs[b + 1]
        if q1 <= q0:
            continue
        slot = int(seq_slots[b])
        old = torch.zeros(taps - 1, h.shape[1], dtype=h.dtype, device=h.device)
        if slot >= 0 and taps > 1 and int(positions[q0]) > 0:
            old = state[slot]
        ext = torch.cat([old, h[q0:q1]], 0)
        acc = h[q0:q1].float() if bias is None else bias.expand(q1 - q0, -1)
        for j in range(taps):
            acc = acc + w[j].float() * ext[j:j + q1 - q0].float()
        out[q0:q1] = (acc if bias is None else F.silu(acc)).to(h.dtype)
        if slot >= 0 and taps > 1:
            state[slot] = ext[q1 - q0:].clone()
    return out


def mingru(zxg, zb, xb, state, seq_slots, positions, q_start, single=False):
    """S_t = (1 - z) S_(t-1) + z c, y = S silu(g) over zxg = [z | x | gate] pre-activations; ``state`` [n, W] fp32."""
    W = zb.shape[0]
    z = torch.sigmoid(zxg[:, :W].float() + zb)
    u = zxg[:, W:2 * W].float() + xb
    c = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    g = F.silu(zxg[:, 2 * W:3 * W].float())
    y = torch.empty(zxg.shape[0], W, dtype=zxg.dtype, device=zxg.device)
    qs = q_start.tolist()
    for b in range(len(qs) - 1):
        q0, q1 = qs[b], qs[b + 1]
        if q1 <= q0:
            continue
        slot = int(seq_slots[b])
        s = state[slot].clone() if slot >= 0 and int(positions[q0]) > 0 else torch.zeros(W, device=zxg.device)
        for t in range(q0, q1):
            s = (1 - z[t]) * s + z[t] * c[t]
            y[t] = (s * g[t]).to(y.dtype)
        if slot >= 0:
            state[slot] = s
    return y


# ---- mixers with a matrix state per head (csrc/kernels/state_mix.cu) ------------------------------------------------------------------
def _softplus(x):
    return F.softplus(x, threshold=1e9)


def state_mix(m, proj, dec_in, gate, conv_state, state, seq_slots, positions, q_start, single, out, extra=None):
    """Runs the mixer described by ``m`` (``ops.specs.StateMix``) over a batch; result columns go to ``out`` [T, H * V]."""
    H, K, V, Hk = m.heads, m.dim, m.vdim, m.heads // m.rep
    qs = q_start.tolist()
    for b in range(len(qs) - 1):
        q0, q1 = qs[b], qs[b + 1]
        if q1 <= q0:
            continue
        slot, n, p0 = int(seq_slots[b]), q1 - q0, int(positions[q0])
        x = proj[q0:q1].float().clone()
        if m.taps:
            c0, nc = m.conv0, m.conv_w.shape[1]
            old = torch.zeros(m.taps - 1, nc, device=proj.device)
            for d in range(1, m.taps):                            # ring row p % taps holds position p's inputs
                if slot >= 0 and p0 - d >= 0:
                    old[m.taps - 1 - d] = conv_state[slot, (p0 - d) % m.taps].float()
            ext = torch.cat([old, x[:, c0:c0 + nc]], 0)
            acc = torch.zeros(n, nc, device=proj.device) if m.conv_b is None else m.conv_b.expand(n, nc).clone()
            for j in range(m.taps):
                acc += m.conv_w[j] * ext[j:j + n]
            if slot >= 0:
                for d in range(1, min(n, m.taps - 1) + 1):
                    conv_state[slot, (p0 + n - d) % m.taps] = proj[q1 - d, c0:c0 + nc]
            x[:, c0:c0 + nc] = F.silu(acc)
        cols = lambda off, h, w: x[:, off:off + h * w].view(n, h, w)          # noqa: B023,E731
        q, k, v = cols(m.q_off, Hk, K), cols(m.k_off, Hk, K), cols(m.v_off, H, V)
        s = torch.ones(n, H, device=proj.device)
        if m.kind == "hgrn":
            z = (dec_in[q0:q1].float() + m.bias).view(n, H, K)
            low = m.lower.view(H, K)
            dec, k, q = low + (1 - low) * torch.sigmoid(z), (1 - low) * torch.sigmoid(-z), F.silu(q)
        if m.kind == "mlstm":
            i, f = (m.gate_cap * torch.tanh((dec_in[q0:q1].float() + m.bias) / m.gate_cap)).view(n, 2, H).unbind(1)
            f, t0 = F.logsigmoid(f), extra[slot, :, K].clone() if slot >= 0 and p0 > 0 else torch.zeros(H, device=proj.device)
            tops, dec = torch.empty(n, H, device=proj.device), torch.empty(n, H, 1, device=proj.device)
            for t in range(n):
                tops[t] = torch.maximum(f[t] + t0, i[t])
                dec[t, :, 0], s[t], t0 = torch.exp(f[t] + t0 - tops[t]), torch.exp(i[t] - tops[t]), tops[t]
            v = torch.cat([v, torch.ones(n, H, 1, device=proj.device)], 2)                # one more column: what the keys add up to
        if m.kind == "delta":
            q, k = (y / torch.sqrt(y.pow(2).sum(-1, keepdim=True) + 1e-6) for y in (q, k))
            s = torch.sigmoid(x[:, m.s_off:m.s_off + H])
        if m.kind == "ssd":
            s = _softplus(x[:, m.s_off:m.s_off + H] + m.bias)
            dec = torch.exp(m.neg_a * s)[..., None]
        elif m.kind in ("delta", "linear"):
            z = dec_in[q0:q1].float() + m.bias
            dec = torch.exp(m.neg_a[:, None] * _softplus(z).view(n, H, K)) if m.kind == "delta" else \
                torch.exp(-m.inv_tau * _softplus(-z)).view(n, H, K)
        q, k = (q * m.q_scale).repeat_interleave(m.rep, 1), k.repeat_interleave(m.rep, 1)
        S = torch.zeros(H, K, v.shape[2], device=proj.device)
        if slot >= 0 and p0 > 0:
            S[..., :V] = state[slot]
            if m.kind == "mlstm":
                S[..., V] = extra[slot, :, :K]
        o = torch.empty(n, H, v.shape[2], device=proj.device)
        for t in range(n):
            S = S * dec[t][..., None]
            u = v[t] - torch.einsum("hkv,hk->hv", S, k[t]) if m.kind == "delta" else v[t]
            S = S + k[t][..., None] * (s[t][:, None] * u)[:, None, :]
            o[t] = torch.einsum("hkv,hk->hv", S, q[t])
        if slot >= 0:
            state[slot] = S[..., :V]
            if m.kind == "mlstm":
                extra[slot, :, :K], extra[slot, :, K] = S[..., V], t0
        if m.kind == "mlstm":
            o = o[..., :V] / (torch.maximum(o[..., V].abs(), torch.exp(-tops)) + 1e-6)[..., None]
            o = (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + m.eps)).reshape(n, H * V)
            out[q0:q1, :H * V] = (o * m.norm_w * torch.sigmoid(gate[q0:q1, :H * V].float()) * m.out_scale).to(out.dtype)
            continue
        if m.kind == "hgrn":
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + m.eps) * m.norm_w
            out[q0:q1, :H * V] = (o * m.out_scale).reshape(n, H * V).to(out.dtype)
            continue
        g = gate[q0:q1, :H * V].float()
        if m.kind == "ssd":
            y = (o + m.skip[:, None] * v).reshape(n, H * V) * F.silu(g)
            y = y.view(n, m.norm_groups, -1)
            y = (y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + m.eps)).reshape(n, H * V) * m.norm_w
        else:
            y = (o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + m.eps) * m.norm_w).reshape(n, H * V)
            y = y * (torch.sigmoid(g) if m.kind == "delta" else F.silu(g))
        out[q0:q1, :H * V] = (y * m.out_scale).to(out.dtype)
    return out


# ---- selective scan (csrc/kernels/selective_scan.cu) ------------------------------------------------------------------------------------
def selective_scan(m, x, z, bc, dt, state, seq_slots, positions, q_start, single, out):
    """Runs the recurrence of ``m`` (``ops.specs.SelectiveScan``) over a batch; result columns go to ``out`` [T, channels]."""
    N = m.state
    qs = q_start.tolist()
    for b in range(len(qs) - 1):
        q0, q1 = qs[b], qs[b + 1]
        if q1 <= q0:
            continue
        slot = int(seq_slots[b])
        S = state[slot].clone() if slot >= 0 and int(positions[q0]) > 0 else torch.zeros_like(m.neg_a)
        xs, BC, d = x[q0:q1].float(), bc[q0:q1].float(), _softplus(dt[q0:q1].float() + m.dt_bias)
        a, u = torch.exp(d[..., None] * m.neg_a), (d * xs)[..., None] * BC[:, None, :N]
        y = torch.empty_like(xs)
        for t in range(q1 - q0):
            S = a[t] * S + u[t]
            y[t] = S @ BC[t, N:2 * N]
        if slot >= 0:
            state[slot] = S
        out[q0:q1] = ((y + m.skip * xs) * F.silu(z[q0:q1].float()) * m.out_scale).to(out.dtype)
    return out


# ---- grouped-query attention over paged rows (csrc/kernels/gqa_attention.cu) ------------------------------------------------------------
def pooled_row(table, b, pool: int, per_block: int, block_size: int):
    """Rows of the pooled tensor that hold the means of blocks ``b`` of ``pool`` positions: they lie in the cache block of their last position."""
    page = (b * pool + pool - 1) // block_size
    return table.long()[page] * per_block + b - page * block_size // pool


def gqa_qkv_post(m, q, k, v, rope_table, positions, slot_mapping, cache, v_first=None, pooled=None):
    """Norms and rotates q and k, stores the rows of the cache; returns q [T, H, D].  ``m``: ``ops.specs.Gqa``."""
    T, H, G, D, V = q.shape[0], m.heads, m.kv_heads, m.dim, m.vdim
    cs = rope_table[positions.long()]

    def post(x, n, w):
        x = x.float().reshape(T, n, D)
        if w is not None:
            x = x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + m.eps) * w
        x = torch.cat([_rope(x[..., :m.rot], cs, not m.neighbours), x[..., m.rot:]], -1)
        return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + m.eps) if m.unit else x
    qo = post(q, H, m.q_norm).to(q.dtype)
    if m.v_mix is not None:
        v = (1 - m.v_mix) * v.float() + m.v_mix * v_first.float()
    rows = torch.cat([post(k, G, m.k_norm).reshape(T, G * D), v.float()], 1).to(cache.dtype)
    ok = slot_mapping >= 0
    cache[slot_mapping[ok].long()] = rows[ok]
    if m.pool:
        pool, tables, seq_lens, q_start, bs, _ = pooled
        P, qs, sl = m.pool, q_start.tolist(), seq_lens.tolist()
        for s in range(len(qs) - 1):
            n, S = qs[s + 1] - qs[s], sl[s]
            for b in range((S - n) // P, S // P) if n > 0 and S > 0 else ():          # blocks that end among the new positions
                pos = torch.arange(b * P, b * P + P, device=cache.device)
                rows = cache[tables[s].long()[pos // bs] * bs + pos % bs].float()
                pool[pooled_row(tables[s], torch.tensor(b, device=cache.device), P, m.pool_rows(bs), bs)] = rows.mean(0).to(pool.dtype)
    return qo


def gqa_attention(m, q, cache, gate, block_tables, seq_lens, q_start, block_size, max_q_len, meta, out, pool=None):
    """Result columns go to ``out`` [T, H * V]; ``gate`` [T, H] pre-activations (``gate_each``: [T, H * V])."""
    T, H, D = q.shape
    G, V = m.kv_heads, m.vdim
    qs, sl = q_start.tolist(), seq_lens.tolist()
    for b in range(len(qs) - 1):
        q0, q1, S = qs[b], qs[b + 1], sl[b]
        if q1 <= q0 or S <= 0:
            continue
        pos = torch.arange(S, device=q.device)
        rows = cache[block_tables[b].long()[pos // block_size] * block_size + pos % block_size].float()
        i, j = torch.arange(S - (q1 - q0), S, device=q.device)[:, None], pos[None]
        see = j <= i
        if m.window:
            see = see & (i - j < m.window)
        if m.chunk:
            see = see & (i // m.chunk == j // m.chunk)
        if m.pool and m.window and S // m.pool:
            blocks = torch.arange(S // m.pool, device=q.device)
            rows = torch.cat([rows, pool[pooled_row(block_tables[b], blocks, m.pool, m.pool_rows(block_size), block_size)].float()])
            see = torch.cat([see, blocks[None] * m.pool + m.pool - 1 <= i - m.window], 1)
        k = rows[:, :G * D].view(-1, G, D).repeat_interleave(H // G, 1)
        v = rows[:, G * D:].view(-1, G, V).repeat_interleave(H // G, 1)
        s = torch.einsum("ihd,jhd->hij", q[q0:q1].float(), k) * m.scale
        if m.softcap:
            s = m.softcap * torch.tanh(s / m.softcap)
        s = s.masked_fill(~see, float("-inf"))
        if m.sink:                                                # a key without a value
            k0 = torch.zeros_like(s[..., :1])
            s = torch.cat([s, k0 if m.sink_w is None else k0 + m.sink_w[:, None, None]], -1)
        p = torch.softmax(s, -1)[..., :rows.shape[0]]
        o = torch.einsum("hij,jhv->ihv", p, v)
        if gate is not None:
            g = torch.sigmoid(gate[q0:q1].float())
            o = o * (g.view(q1 - q0, H, V) if m.gate_each else g[..., None])
        out[q0:q1, :H * V] = (o * m.out_scale).reshape(q1 - q0, H * V).to(out.dtype)
    return out
