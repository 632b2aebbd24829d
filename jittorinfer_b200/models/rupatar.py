"""Rupatar: a decoder of windowed attention with pooled blocks, HGRN2 and mLSTM layers, each followed by a mixture of experts.

Both sublayers of a layer read a norm in groups (equal parts of the row, each over its own root mean square) of one fp32 residual row:
``x <- x + mixer(norm1(x))``, then ``x <- x + ff(norm2(x))`` (a layer may have no feed-forward).  What the layers are made of:

* **attention** -- grouped queries (biases on q, k, v and the output, neighbouring dimensions rotated by stretched angles, q and k over their
  root mean square after it), a sliding window and beside it one mean key and value per block of positions that has left it, a sink of score
  0, a gate per channel; layers marked for it cache a blend of their values and those of the first such layer;
* **hgrn2** -- linear attention whose forget gate, bounded from below per channel, is also what the keys are made of (k = 1 - f);
* **mlstm** -- a matrix memory with exponential gates relative to a running maximum, normalised by what the keys add up to;
* **feed-forward** -- experts without gates (exact gelu), sigmoid scores that are not renormalised and multiply the experts' input, a shared
  expert.

The recurrences are two kinds of ``ops.state_mix``.  Attention rows and the pooled rows are paged; states and the running maxima live in one
row per sequence slot (``runtime/cache.py:HybridCache``), and a batch range that starts at position 0 starts from zeros.

Every mixer reads one product of its input with its stacked projections (columns in multiples of 8, attention's biases as its epilogue).  A
shared expert joins the grouped expert products when its width is a
multiple of theirs.  On a GPU a decode step runs per layer: input GEMM, the mixer's launches, output GEMM, ``scaled_update``
(residual, norm), router, gating, expert sort, two grouped GEMMs, ``scaled_update`` (combine, residual, next norm).  ``dtype`` float32 runs the
same graph with fp32 kernels.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Dict, Iterable, Iterator, List, Optional, Tuple

import torch

from .. import ops
from ..ops.specs import Gqa, RowNorms, StateMix
from ..utils import trace as _trace
from .deepseek2 import ForwardBatch
from .folder import Rotation, checked_tensors, fits, rope_table, stack_rows, up
from .weights import ShardSpec, _stream_seed

ARCH = "Rupatar"
MAX_EXPERTS, MAX_CHOICES, MAX_GROUPS = 256, 32, 1024         # what the routing and row kernels are built for


# ---- configuration -----------------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class AttentionMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: int                    # 0: none
    pool: int                      # positions of a pooled block, 0: none
    rot: Rotation
    v_mix: bool = False


@dataclass(frozen=True)
class Hgrn2Mixer:
    heads: int
    dim: int
    vdim: int


@dataclass(frozen=True)
class MlstmMixer:
    heads: int
    dim: int
    vdim: int
    gate_cap: float


@dataclass(frozen=True)
class Experts:
    ff: int
    experts: int
    top: int
    shared: Optional[int] = None   # width of the shared expert


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                     # AttentionMixer | Hgrn2Mixer | MlstmMixer
    mlp: Optional[Experts]


def _mixer(kind: str, m: Dict[str, Any]):
    sizes = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    if min(sizes) < 1:
        raise ValueError("heads and their sizes are at least 1")
    if kind == "hgrn2":
        return Hgrn2Mixer(*sizes)
    if kind == "mlstm":
        return MlstmMixer(*sizes, float(m["gate_cap"]))
    if kind != "attention":
        raise ValueError(f"unknown mixer {kind!r}")
    mask, r = m.get("mask") or {}, m["rot"]
    a = AttentionMixer(sizes[0], int(m["kv_heads"]), *sizes[1:], float(m["scale"]), int(mask.get("size") or 0), int(mask.get("pool") or 0),
                       Rotation(int(r["dims"]), float(r["base"]), stretch=float((r.get("scaling") or {}).get("factor") or 1.0)), bool(m.get("v_mix")))
    if a.heads % a.kv_heads or a.rot.dims % 2 or a.rot.dims > a.dim:
        raise ValueError("heads must be a multiple of kv_heads, the rotated dimensions an even part of the head")
    if min(a.window, a.pool) < 0 or a.pool and not a.window:
        raise ValueError("pooled blocks are what lies before a window")
    return a


def _mixer_config(x) -> Tuple[str, Dict[str, Any]]:
    if isinstance(x, Hgrn2Mixer):
        return "hgrn2", dict(heads=x.heads, dim=x.dim, vdim=x.vdim)
    if isinstance(x, MlstmMixer):
        return "mlstm", dict(heads=x.heads, dim=x.dim, vdim=x.vdim, gate_cap=x.gate_cap)
    return "attention", dict(heads=x.heads, kv_heads=x.kv_heads, dim=x.dim, vdim=x.vdim, scale=x.scale, mask=dict(size=x.window, pool=x.pool),
                             rot=dict(base=x.rot.base, dims=x.rot.dims, scaling=dict(factor=x.rot.stretch)), v_mix=x.v_mix)


def _mlp(m: Optional[Dict[str, Any]]) -> Optional[Experts]:
    if m is None:
        return None
    if m.get("kind") != "moe":
        raise ValueError(f"unknown feed-forward {m.get('kind')!r}")
    r, sh = m["router"], m.get("shared")
    x = Experts(int(m["expert"]["ff"]), int(r["experts"]), int(r["top"]), None if sh is None else int(sh["ff"]))
    if not 1 <= x.experts <= MAX_EXPERTS or not 1 <= x.top <= min(x.experts, MAX_CHOICES):
        raise ValueError(f"top {x.top} of {x.experts} experts: at most {MAX_CHOICES} of {MAX_EXPERTS}")
    return x


@dataclass
class RupatarHParams:
    n_vocab: int
    n_embd: int
    eps: float
    groups: int
    embed_scale: float
    layers: List[LayerSpec] = field(default_factory=list)
    bos_id: int = -1               # token ids only: the design names no special tokens
    eos_id: int = -1
    n_ctx_train: int = 1 << 20

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @property
    def first_mix(self) -> int:
        """The layer whose values the later value-mixing layers blend in, -1: none."""
        return next((i for i, L in enumerate(self.layers) if isinstance(L.mixer, AttentionMixer) and L.mixer.v_mix), -1)

    @classmethod
    def from_config(cls, cfg: Dict[str, Any]) -> "RupatarHParams":
        if cfg.get("architecture") != ARCH:
            raise ValueError(f"architecture {cfg.get('architecture')!r} is not {ARCH}")
        layers: List[LayerSpec] = []
        for i, e in enumerate(cfg["layers"]):
            try:
                layers.append(LayerSpec(_mixer(e["type"], e["mixer"]), _mlp(e.get("mlp"))))
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
        hp = cls(n_vocab=int(cfg["vocab"]), n_embd=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), groups=int(cfg["norm"]["groups"]),
                 embed_scale=float(cfg["embedding"]["scale"]), layers=layers)
        if not 1 <= hp.groups <= MAX_GROUPS or hp.n_embd % hp.groups:
            raise ValueError(f"norms of {hp.groups} equal parts (at most {MAX_GROUPS}) over a width of {hp.n_embd}")
        mixed = {(L.mixer.kv_heads, L.mixer.vdim) for L in layers if isinstance(L.mixer, AttentionMixer) and L.mixer.v_mix}
        if len({g * v for g, v in mixed}) > 1:
            raise ValueError("layers that mix values hold as many of them as the first")
        return hp

    def to_config(self) -> Dict[str, Any]:
        out = []
        for L in self.layers:
            kind, mix = _mixer_config(L.mixer)
            m, mlp = L.mlp, None
            if m is not None:
                mlp = dict(kind="moe", expert=dict(ff=m.ff), router=dict(experts=m.experts, top=m.top))
                if m.shared is not None:
                    mlp["shared"] = dict(ff=m.shared)
            out.append(dict(type=kind, mixer=mix, mlp=mlp))
        return dict(architecture=ARCH, vocab=self.n_vocab, width=self.n_embd, norm=dict(eps=self.eps, groups=self.groups),
                    embedding=dict(scale=self.embed_scale), layers=out)

    def n_params(self) -> int:
        return sum(math.prod(s) for s in tensor_table(self).values())


def preset(name: str) -> RupatarHParams:
    """Named shapes for tests, examples and benchmarks (random weights)."""
    name = name.lower().replace("_", "-")

    def stack(n, attn, hgrn, mlstm, mlp):
        return [LayerSpec((attn, hgrn, attn, mlstm)[i % 4], mlp) for i in range(n)]
    if name == "rupatar-tiny":
        attn = AttentionMixer(6, 2, 40, 24, 0.2, 40, 6, Rotation(24, 10000.0, stretch=2.0), True)
        return RupatarHParams(n_vocab=600, n_embd=160, eps=1e-5, groups=5, embed_scale=2.0,
                              layers=stack(4, attn, Hgrn2Mixer(3, 40, 24), MlstmMixer(4, 24, 40, 10.0), Experts(64, 10, 3, 64)))
    if name in ("rupatar-lite", "rupatar-v2"):
        # the layer sizes of DeepSeek-V2-Lite (64 experts of which 6 run) and DeepSeek-V2 (160 experts), two shared experts' width
        w, n, mlp = (2048, 12, Experts(1408, 64, 6, 2816)) if name == "rupatar-lite" else (5120, 4, Experts(1536, 160, 6, 3072))
        h = w // 128
        attn = AttentionMixer(h, h // 4, 128, 128, 128 ** -0.5, 512, 16, Rotation(64, 500000.0, stretch=4.0), True)
        return RupatarHParams(n_vocab=102400, n_embd=w, eps=1e-6, groups=8, embed_scale=1.0,
                              layers=stack(n, attn, Hgrn2Mixer(h, 128, 128), MlstmMixer(h, 128, 128, 15.0), mlp))
    raise KeyError(name)


# ---- weights -------------------------------------------------------------------------------------------------------------------
def tensor_table(hp: RupatarHParams) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint tensor name -> shape."""
    d = hp.n_embd
    t: Dict[str, Tuple[int, ...]] = {"embed": (hp.n_vocab, d)}
    for i, L in enumerate(hp.layers):
        p, x, m = f"l{i}.", L.mixer, L.mlp
        for k in ("norm1",) + (("norm2",) if m is not None else ()):
            t[p + k] = (d,)
        p += "mix."
        n = x.heads * x.dim
        if isinstance(x, AttentionMixer):
            for k, rows in (("q", n), ("k", x.kv_heads * x.dim), ("v", x.kv_heads * x.vdim)):
                t.update({p + k: (rows, d), p + k + ".b": (rows,)})
            if x.v_mix:
                t[p + "vmix"] = ()
            t.update({p + "g": (x.heads * x.vdim, d), p + "o.b": (d,)})
        elif isinstance(x, Hgrn2Mixer):
            t.update({p + "q": (n, d), p + "f": (n, d), p + "f.b": (n,), p + "lower": (n,), p + "v": (x.heads * x.vdim, d), p + "norm": (x.vdim,)})
        else:
            t.update({p + "q": (n, d), p + "k": (n, d), p + "v": (x.heads * x.vdim, d), p + "g": (x.heads * x.vdim, d), p + "norm": (x.heads * x.vdim,)})
            for k in "if":
                t.update({p + k: (x.heads, d), p + k + ".b": (x.heads,)})
        t[p + "o"] = (d, x.heads * x.vdim)
        if m is not None:
            p = f"l{i}.mlp."
            for e, ff in [(f"e{j}", m.ff) for j in range(m.experts)] + ([("shared", m.shared)] if m.shared is not None else []):
                t.update({p + e + ".up": (ff, d), p + e + ".down": (d, ff)})
            t[p + "router"] = (m.experts, d)
    t["final.norm"] = (d,)
    t["head"] = (hp.n_vocab, d)
    return t


def _unused(hp: RupatarHParams, name: str) -> bool:
    """The norm of a feed-forward the layer does not have, the blend of a layer that mixes no values."""
    layer, _, k = name.partition(".")
    if not (layer[1:].isdigit() and int(layer[1:]) < hp.n_layer):
        return False
    L = hp.layers[int(layer[1:])]
    return k == "norm2" and L.mlp is None or k == "mix.vmix" and not getattr(L.mixer, "v_mix", False)


def iter_checkpoint(directory: str, hp: RupatarHParams) -> Iterator[Tuple[str, torch.Tensor]]:
    """(name, CPU tensor) of every tensor of the model from the folder's safetensors file(s); checks names and shapes."""
    return checked_tensors(directory, tensor_table(hp), lambda n: _unused(hp, n))


def iter_random(hp: RupatarHParams, seed: int = 0, dtype: torch.dtype = torch.float32, device="cpu") -> Iterator[Tuple[str, torch.Tensor]]:
    """Random weights: matrices N(0, 1 / fan-in), norms around one, forget gates of a few to a few hundred tokens."""
    dev = torch.device(device)
    gen = torch.Generator(device=dev)
    for name, shape in tensor_table(hp).items():
        gen.manual_seed(_stream_seed(seed, name, 0))
        leaf = name.rsplit(".", 1)[-1]
        std = 1.0 if name == "embed" or leaf == "lower" else 0.2 if len(shape) < 2 else shape[1] ** -0.5
        x = torch.empty(shape, dtype=dtype, device=dev).normal_(0.0, std, generator=gen)
        yield name, x + 1 if "norm" in leaf else torch.sigmoid(x) if leaf == "lower" else x + 0.5 if leaf == "vmix" else x + 3 if name.endswith("mix.f.b") else x


def load_config(directory: str) -> RupatarHParams:
    with open(os.path.join(directory, "config.json")) as f:
        return RupatarHParams.from_config(json.load(f))


class _Layer:
    __slots__ = ("norm1", "norm2", "w_in", "b_in", "cols", "w_o", "b_o", "attn", "rope", "mix", "router", "n_merged", "w_up_exps",
                 "w_down_exps", "w_up_sh", "w_down_sh")

    def __init__(self):
        for s in self.__slots__:
            setattr(self, s, None)


# ---- model -----------------------------------------------------------------------------------------------------------------------
class RupatarModel:
    recurrent = True                  # sequences carry a state besides their cached rows (see Scheduler.set_recurrent)
    split = False
    comm = None

    def __init__(self, hp: RupatarHParams, weights: Iterable[Tuple[str, torch.Tensor]], dtype: torch.dtype = torch.bfloat16, device="cpu",
                 max_positions: int = 8192, block_size: int = 64):
        self.hp, self.dtype, self.device = hp, dtype, torch.device(device)
        self.spec = ShardSpec()
        self.block_size, self.max_positions = block_size, max_positions
        self.tensor_hook = None       # called as tensor_hook(name, tensor) with every layer's residual; steps then run eagerly
        self.layers = [_Layer() for _ in hp.layers]
        tables: Dict[Rotation, torch.Tensor] = {}
        for L, s in zip(self.layers, hp.layers):
            if isinstance(s.mixer, AttentionMixer):
                rot = s.mixer.rot
                if rot not in tables:
                    tables[rot] = rope_table(max_positions, rot, self.device)
                L.rope = tables[rot]
        self._load(weights)

    # ---- weight intake ---------------------------------------------------------------------------------------------------------
    def _load(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> None:
        hp, dev, f32 = self.hp, self.device, torch.float32
        table, seen = tensor_table(hp), set()
        pend: Dict[str, torch.Tensor] = {}
        todo = [set(k for k in table if k.startswith(f"l{i}.")) for i in range(hp.n_layer)]
        for name, t in weights:
            _trace.log_tensor(name, t.shape, t.dtype, "")
            if name not in table:
                if _unused(hp, name):
                    continue
                raise KeyError(f"unknown tensor {name}")
            if not fits(t.shape, table[name]):
                raise ValueError(f"{name}: shape {tuple(t.shape)} != expected {table[name]}")
            seen.add(name)
            layer, _, base = name.partition(".")
            i = int(layer[1:]) if layer[0] == "l" and layer[1:].isdigit() else -1
            if i >= 0 and base.startswith("mlp.") and base.count(".") == 2:
                self._take_expert(i, *base.split(".")[1:], t)          # straight into the stacked tensors: nothing is held twice
            else:
                pend[name] = t.to(device=dev, dtype=f32 if t.dim() < 2 else self.dtype).contiguous()
            if i >= 0:
                todo[i].discard(name)
                if not todo[i]:                               # complete: stack it and let the parts go
                    self._finish_layer(i, pend)
        missing = [n for n in table if n not in seen]
        if missing:
            raise ValueError(f"missing tensors: {len(missing)}, e.g. {missing[:3]}")
        self.embed, self.final_norm, self.head = pend.pop("embed"), pend.pop("final.norm"), pend.pop("head")

    def _take_expert(self, i: int, who: str, kind: str, t: torch.Tensor) -> None:
        L, m, d = self.layers[i], self.hp.layers[i].mlp, self.hp.n_embd
        if L.n_merged is None:            # a shared expert as wide as n routed ones is a sum over n experts of that width
            n = m.shared // m.ff if m.shared is not None and m.shared % m.ff == 0 else 0
            L.n_merged = n if m.experts + n <= MAX_EXPERTS and m.top + n <= MAX_CHOICES else 0
            for k, s in (("up", (m.ff, d)), ("down", (d, m.ff))):
                setattr(L, f"w_{k}_exps", torch.empty((m.experts + L.n_merged,) + s, dtype=self.dtype, device=self.device))
        w = getattr(L, f"w_{kind}_exps")
        if who != "shared":
            w[int(who[1:])].copy_(t)
        elif L.n_merged:
            w[m.experts:].copy_(t.reshape(L.n_merged, m.ff, d) if kind == "up" else t.reshape(d, L.n_merged, m.ff).transpose(0, 1))
        else:
            setattr(L, f"w_{kind}_sh", t.to(device=self.device, dtype=self.dtype).contiguous())

    def _finish_layer(self, i: int, pend: Dict[str, torch.Tensor]) -> None:
        L, s, eps = self.layers[i], self.hp.layers[i], self.hp.eps
        take = lambda k: pend.pop(f"l{i}.{k}")                                  # noqa: E731
        x = s.mixer
        L.norm1 = take("norm1")
        if s.mlp is not None:
            L.norm2, L.router = take("norm2"), take("mlp.router")
        if isinstance(x, MlstmMixer):
            parts = [(k, take("mix." + k)) for k in "qkvg"] + [("gates", torch.cat([take("mix.i"), take("mix.f")]))]
        else:
            parts = [(k, take("mix." + k)) for k in ("qfv" if isinstance(x, Hgrn2Mixer) else "qkvg")]
        L.w_in, c = stack_rows(parts)
        L.cols, w = c, take("mix.o")
        L.w_o = torch.zeros(w.shape[0], up(w.shape[1]), dtype=w.dtype, device=w.device)      # its input's rows are 16-byte multiples
        L.w_o[:, :w.shape[1]] = w
        if isinstance(x, AttentionMixer):
            L.b_in, L.b_o = torch.zeros(L.w_in.shape[0], dtype=torch.float32, device=self.device), take("mix.o.b")
            for k in "qkv":
                b = take(f"mix.{k}.b")
                L.b_in[c[k]:c[k] + b.shape[0]] = b
            lam = float(take("mix.vmix")) if x.v_mix else None
            L.attn = Gqa(x.heads, x.kv_heads, x.dim, x.vdim, x.rot.dims, x.scale, window=x.window, sink=True, eps=eps, neighbours=True, unit=True, pool=x.pool,
                         v_mix=None if i == self.hp.first_mix else lam, gate_each=True)
        elif isinstance(x, Hgrn2Mixer):
            L.mix = StateMix("hgrn", x.heads, x.dim, x.vdim, q_off=c["q"], v_off=c["v"], bias=take("mix.f.b"), lower=take("mix.lower"),
                             norm_w=take("mix.norm"), eps=eps)
        else:
            L.mix = StateMix("mlstm", x.heads, x.dim, x.vdim, q_off=c["q"], k_off=c["k"], v_off=c["v"], bias=torch.cat([take("mix.i.b"), take("mix.f.b")]), norm_w=take("mix.norm"), q_scale=x.dim ** -0.5,
                             gate_cap=x.gate_cap, eps=eps)

    def weight_bytes(self) -> int:
        ts = [self.embed, self.final_norm, self.head]
        for L in self.layers:
            ts += [getattr(L, k) for k in L.__slots__] + [v for x in (L.mix,) if x is not None for v in vars(x).values()]
        return sum(t.numel() * t.element_size() for t in ts if isinstance(t, torch.Tensor))

    # ---- cache -------------------------------------------------------------------------------------------------------------------
    def cache_bytes_per_token(self) -> int:
        el, bs = torch.empty(0, dtype=self.dtype).element_size(), self.block_size
        return sum(L.attn.kv_row * el * (bs + L.attn.pool_rows(bs)) // bs for L in self.layers if L.attn is not None)

    def make_cache(self, n_slots: int, n_seqs: int):
        """Paged rows of ``n_slots`` tokens (and pooled rows beside them) for the attention, a state row per sequence slot for the recurrences."""
        from ..runtime.cache import HybridCache
        mixes = [L.mix for L in self.layers]
        state = {"mix": [m and ((m.heads, m.dim, m.vdim), torch.float32) for m in mixes],
                 "extra": [((m.heads, m.dim + 1), torch.float32) if m is not None and m.kind == "mlstm" else None for m in mixes]}
        return HybridCache([L.attn and L.attn.kv_row for L in self.layers], state, n_slots, n_seqs, self.dtype, self.device, self.block_size,
                           [L.attn.pool_rows(self.block_size) if L.attn is not None else 0 for L in self.layers])

    # ---- forward -----------------------------------------------------------------------------------------------------------------
    def _attention(self, i: int, L: _Layer, h: torch.Tensor, b: ForwardBatch, cache, single: bool, v_first) -> Tuple[torch.Tensor, Any]:
        T, c, a = h.shape[0], L.cols, L.attn
        proj = ops.linear(h, L.w_in, residual=L.b_in.expand(T, -1))
        v = proj[:, c["v"]:c["v"] + a.kv_heads * a.vdim]
        if i == self.hp.first_mix:
            v_first = v
        pooled = (cache.pool[i], b.block_tables, b.seq_lens, b.q_start, self.block_size, single) if a.pool else None
        q = ops.gqa_qkv_post(a, proj[:, c["q"]:c["q"] + a.heads * a.dim], proj[:, c["k"]:c["k"] + a.kv_heads * a.dim], v, L.rope, b.positions,
                             b.slot_mapping, cache[i], v_first, pooled)
        n = a.heads * a.vdim
        y = self._rows(h, L, n)
        ops.gqa_attention(a, q, cache[i], proj[:, c["g"]:c["g"] + n], b.block_tables, b.seq_lens, b.q_start, self.block_size, b.max_q_len, b.attn_meta, y[:, :n],
                          cache.pool[i])
        return ops.linear(y, L.w_o, residual=L.b_o.expand(T, -1)), v_first

    def _recurrence(self, i: int, L: _Layer, h: torch.Tensor, b: ForwardBatch, cache, single: bool) -> torch.Tensor:
        c, m = L.cols, L.mix
        n = m.heads * m.vdim
        proj = ops.linear(h, L.w_in)
        if m.kind == "hgrn":
            dec, gate = proj[:, c["f"]:c["f"] + m.heads * m.dim], None
        else:
            dec, gate = proj[:, c["gates"]:c["gates"] + 2 * m.heads], proj[:, c["g"]:c["g"] + n]
        y = self._rows(h, L, n)
        ops.state_mix(m, proj, dec, gate, None, cache.state["mix"][i], b.seq_slots, b.positions, b.q_start, single, y[:, :n], cache.state["extra"][i])
        return ops.linear(y, L.w_o)

    @staticmethod
    def _rows(h: torch.Tensor, L: _Layer, n: int) -> torch.Tensor:
        """Where a mixer's ``n`` result columns go; columns nobody writes are zero."""
        return (torch.zeros if L.w_o.shape[1] > n else torch.empty)(h.shape[0], L.w_o.shape[1], dtype=h.dtype, device=h.device)

    def _ff(self, L: _Layer, m: Experts, h: torch.Tensor) -> Dict[str, Any]:
        """The feed-forward's part of ``ops.scaled_update``'s arguments."""
        ids, wts = ops.moe_gate(h, L.router, None, m.top, 1, 1, 1.0, False, True, L.n_merged)
        y, dest = ops.moe_routed(h, ids, wts, None, L.w_up_exps, L.w_down_exps)
        out: Dict[str, Any] = {"moe": (y, dest, None)}
        if m.shared is not None and not L.n_merged:
            out["dense"] = ops.linear(ops.linear(h, L.w_up_sh, unary=("gelu",)), L.w_down_sh)
        return out

    @torch.no_grad()
    def forward(self, batch: ForwardBatch, cache) -> torch.Tensor:
        """fp32 logits [len(out_rows), n_vocab]; ``cache`` is a ``HybridCache`` of this model."""
        hp, b = self.hp, batch
        single = b.max_q_len == 1 and b.seq_lens.shape[0] == b.tokens.shape[0]       # row t is sequence t's only token
        v_first = None

        def norm(w):                  # what follows a residual update
            return None if w is None else RowNorms(hp.eps, w, groups=hp.groups)

        after = [L.norm1 for L in self.layers[1:]] + [None]
        x, h, _ = ops.embed_norm(self.embed, b.tokens, None, hp.eps, norm(self.layers[0].norm1) if self.layers else None, hp.embed_scale)
        for i, (L, s) in enumerate(zip(self.layers, hp.layers)):
            if L.attn is not None:
                o, v_first = self._attention(i, L, h, b, cache, single, v_first)
            else:
                o = self._recurrence(i, L, h, b, cache, single)
            x, h, _ = ops.scaled_update(x, o, None, nxt=norm(L.norm2 if s.mlp is not None else after[i]))
            if s.mlp is not None:
                x, h, _ = ops.scaled_update(x, None, None, nxt=norm(after[i]), **self._ff(L, s.mlp, h))
            if self.tensor_hook is not None:
                self.tensor_hook(f"blk.{i}.mix_out", o)
                self.tensor_hook(f"blk.{i}.ffn_out", x.clone())
        if b.out_rows.shape[0] == 0:
            return torch.empty(0, hp.n_vocab, dtype=torch.float32, device=self.device)
        xo = ops.rms_rows(x, b.out_rows, self.final_norm, hp.eps, self.dtype, hp.groups)
        logits = ops.linear(xo, self.head, out_dtype=torch.float32)
        if self.tensor_hook is not None:
            self.tensor_hook("result_norm", xo)
            self.tensor_hook("result_output", logits)
        return logits
