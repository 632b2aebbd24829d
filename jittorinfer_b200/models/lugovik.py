"""Lugovik: a decoder whose layers mix tokens by a state-space recurrence, a delta rule, or attention beside gated linear attention.

Both sublayers of a layer stand between two norms over an fp32 residual stream ``x``:
``x <- x + norm(mixer(norm(x)))``, then ``x <- x + norm(ff(norm(x)))`` (a layer may have no feed-forward).  What the layers are made of:

* **mamba2** -- one decay per head, B and C shared by groups of heads, a short convolution ahead of it, a gated norm behind it;
* **channel_delta** -- the gated delta rule with one decay per key channel, convolved and unit-normed q and k;
* **parallel** -- grouped-query attention (normed q and k, YaRN, softcap, chunked mask, sink, a gate per head) and gated linear attention
  on one input, their weighted outputs added;
* **feed-forward** -- gated, tanh form of gelu.

The three recurrences are one mechanism (``ops.state_mix``) with a matrix state per head.  Attention rows are paged; states and the
convolutions' last inputs live in one row per sequence slot (``runtime/cache.py:HybridCache``), and a batch range that starts at
position 0 starts from zeros.

Every mixer reads one product of its input with its stacked projections (columns in multiples of 8, so that any slice can feed the
tensor cores) and its output projections are one product as well: the parallel mixer's halves write their scaled results side by
side.  On a GPU a decode step runs per layer: input GEMM, [low-rank GEMM,] the mixer's launches, output GEMM, ``post_norm`` (norm of the
output, residual, next norm), gate|up GEMM, down GEMM, ``post_norm``.  ``dtype`` float32 runs the same graph with fp32 kernels.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field, replace
from typing import Any, Dict, Iterable, Iterator, List, Optional, Sequence, Tuple

import torch

from .. import ops
from ..ops.specs import Gqa, StateMix
from ..utils import trace as _trace
from .deepseek2 import ForwardBatch
from .folder import Rotation, Yarn, block_diagonal, checked_tensors, fits, rope_table, stack_rows, up
from .weights import ShardSpec, _stream_seed

ARCH = "Lugovik"


# ---- configuration -----------------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class Mamba2Mixer:
    heads: int
    vdim: int
    state: int
    groups: int
    norm_groups: int
    conv: int

    @property
    def inner(self) -> int:
        return self.heads * self.vdim


@dataclass(frozen=True)
class DeltaMixer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    conv: int


@dataclass(frozen=True)
class AttentionPart:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    chunk: int
    rot: Rotation


@dataclass(frozen=True)
class LinearPart:
    heads: int
    dim: int
    vdim: int
    tau: float


@dataclass(frozen=True)
class ParallelMixer:
    left: AttentionPart
    right: LinearPart
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                     # Mamba2Mixer | DeltaMixer | ParallelMixer
    ff: Optional[int]              # width of the feed-forward, None: the layer has none


def _rotation(r: Dict[str, Any]) -> Rotation:
    s = r.get("scaling")
    return Rotation(int(r["dims"]), float(r["base"]),
                    None if s is None else Yarn(float(s["factor"]), float(s["original"]), float(s["fast"]), float(s["slow"])))


def _mixer(kind: str, m: Dict[str, Any]):
    if kind == "mamba2":
        x = Mamba2Mixer(int(m["heads"]), int(m["vdim"]), int(m["state"]), int(m["groups"]), int(m["norm_groups"]), int(m["conv"]))
        if x.heads % x.groups or x.inner % x.norm_groups:
            raise ValueError("heads must be a multiple of groups, their width one of norm_groups")
    elif kind == "channel_delta":
        x = DeltaMixer(int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"]), int(m["conv"]))
        if x.heads % x.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
    elif kind == "parallel":
        a, r = m["left"], m["right"]
        left = AttentionPart(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]), float(a.get("softcap") or 0.0),
                             int((a.get("mask") or {}).get("size") or 0), _rotation(a["rot"]))
        if left.heads % left.kv_heads or left.rot.dims % 2 or left.rot.dims > left.dim:
            raise ValueError("heads must be a multiple of kv_heads, the rotated dimensions an even part of the head")
        x = ParallelMixer(left, LinearPart(int(r["heads"]), int(r["dim"]), int(r["vdim"]), float(r["tau"])),
                          float(m["left_scale"]), float(m["right_scale"]))
    else:
        raise ValueError(f"unknown mixer {kind!r}")
    if getattr(x, "conv", 1) < 1:
        raise ValueError("a convolution has at least one tap")
    return x


def _mixer_config(x) -> Tuple[str, Dict[str, Any]]:
    if isinstance(x, Mamba2Mixer):
        return "mamba2", dict(heads=x.heads, vdim=x.vdim, state=x.state, groups=x.groups, norm_groups=x.norm_groups, conv=x.conv)
    if isinstance(x, DeltaMixer):
        return "channel_delta", dict(heads=x.heads, kv_heads=x.kv_heads, dim=x.dim, vdim=x.vdim, conv=x.conv)
    a, r, y = x.left, x.right, x.left.rot.yarn
    rot: Dict[str, Any] = dict(base=a.rot.base, dims=a.rot.dims)
    if y is not None:
        rot["scaling"] = dict(factor=y.factor, original=y.original, fast=y.fast, slow=y.slow)
    return "parallel", dict(left=dict(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale, softcap=a.softcap,
                                      mask=dict(size=a.chunk), rot=rot),
                            right=dict(heads=r.heads, dim=r.dim, vdim=r.vdim, tau=r.tau), left_scale=x.left_scale, right_scale=x.right_scale)


@dataclass
class LugovikHParams:
    n_vocab: int
    n_embd: int
    eps: float
    embed_scale: float
    layers: List[LayerSpec] = field(default_factory=list)
    random_rank: int = 16          # inner width of the low-rank projections when weights are random (a checkpoint brings its own)
    bos_id: int = -1               # token ids only: the design names no special tokens
    eos_id: int = -1
    n_ctx_train: int = 1 << 20

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @classmethod
    def from_config(cls, cfg: Dict[str, Any]) -> "LugovikHParams":
        if cfg.get("architecture") != ARCH:
            raise ValueError(f"architecture {cfg.get('architecture')!r} is not {ARCH}")
        layers: List[LayerSpec] = []
        for i, e in enumerate(cfg["layers"]):
            try:
                mix, mlp = _mixer(e["type"], e["mixer"]), e.get("mlp")
                if mlp is not None and mlp.get("kind") != "dense":
                    raise ValueError(f"unknown feed-forward {mlp.get('kind')!r}")
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
            layers.append(LayerSpec(mix, None if mlp is None else int(mlp["ff"])))
        return cls(n_vocab=int(cfg["vocab"]), n_embd=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]),
                   layers=layers)

    def to_config(self) -> Dict[str, Any]:
        out = []
        for L in self.layers:
            kind, mix = _mixer_config(L.mixer)
            out.append({"type": kind, "mixer": mix, "mlp": None if L.ff is None else {"kind": "dense", "ff": L.ff}})
        return {"architecture": ARCH, "vocab": self.n_vocab, "width": self.n_embd, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "layers": out}

    def n_params(self) -> int:
        return sum(math.prod(s) for s in _concrete(self).values())


def preset(name: str) -> LugovikHParams:
    """Named shapes for tests, examples and benchmarks (random weights)."""
    name = name.lower().replace("_", "-")

    def stack(n, mamba, delta, par, ff):
        return [LayerSpec((mamba, delta, par, mamba)[i % 4], ff) for i in range(n)]

    def attention(heads, kv, dim, chunk, base):
        return AttentionPart(heads, kv, dim, dim, dim ** -0.5, 30.0, chunk, Rotation(dim, base, Yarn(4.0, 4096, 32.0, 1.0)))
    if name == "lugovik-tiny":
        par = ParallelMixer(replace(attention(6, 2, 40, 48, 10000.0), vdim=24, rot=Rotation(24, 10000.0, Yarn(2.0, 256, 16.0, 1.0))),
                            LinearPart(3, 24, 40, 12.0), 0.8, 1.1)
        return LugovikHParams(n_vocab=640, n_embd=160, eps=1e-5, embed_scale=4.0,
                              layers=stack(4, Mamba2Mixer(6, 24, 16, 2, 3, 4), DeltaMixer(4, 2, 24, 40, 4), par, 208), random_rank=12)
    if name in ("lugovik-lite", "lugovik-wide"):
        # heads of 128: 16 of them at width 2048, 32 at width 4096
        w, n, ff = (2048, 12, 5632) if name == "lugovik-lite" else (4096, 8, 11008)
        h = w // 128
        par = ParallelMixer(attention(h, h // 4, 128, 512, 500000.0), LinearPart(h, 128, 128, 16.0), 0.7, 0.7)
        return LugovikHParams(n_vocab=102400, n_embd=w, eps=1e-6, embed_scale=w ** 0.5,
                              layers=stack(n, Mamba2Mixer(w // 32, 64, 128, 1, 1, 4), DeltaMixer(h, h, 128, 128, 4), par, ff), random_rank=128)
    raise KeyError(name)


# ---- weights -------------------------------------------------------------------------------------------------------------------
def tensor_table(hp: LugovikHParams) -> Dict[str, Tuple[Optional[int], ...]]:
    """Checkpoint tensor name -> shape; None: a low-rank projection's inner width, which only the tensors tell."""
    d = hp.n_embd
    t: Dict[str, Tuple[Optional[int], ...]] = {"embed": (hp.n_vocab, d)}
    for i, L in enumerate(hp.layers):
        p, m = f"l{i}.", L.mixer
        for k in ("norm1", "norm1b") + (("norm2", "norm2b") if L.ff is not None else ()):
            t[p + k] = (d,)
        p += "mix."
        if isinstance(m, Mamba2Mixer):
            ch = m.inner + 2 * m.groups * m.state
            t.update({p + "in": (m.inner + ch + m.heads, d), p + "conv": (ch, m.conv), p + "conv.b": (ch,), p + "dt_bias": (m.heads,),
                      p + "A_log": (m.heads,), p + "D": (m.heads,), p + "norm": (m.inner,), p + "o": (d, m.inner)})
        elif isinstance(m, DeltaMixer):
            for k, n in (("q", m.kv_heads * m.dim), ("k", m.kv_heads * m.dim), ("v", m.heads * m.vdim)):
                t[p + k] = (n, d)
                t[p + k + ".conv"] = (n, m.conv)
            t.update({p + "b": (m.heads, d), p + "A_log": (m.heads,), p + "norm": (m.vdim,), p + "a1": (None, d),
                      p + "a2": (m.heads * m.dim, None), p + "dt_bias": (m.heads * m.dim,), p + "g1": (None, d),
                      p + "g2": (m.heads * m.vdim, None), p + "o": (d, m.heads * m.vdim)})
        else:
            a, r, q = m.left, m.right, p + "left."
            t.update({q + "q": (a.heads * a.dim, d), q + "k": (a.kv_heads * a.dim, d), q + "v": (a.kv_heads * a.vdim, d), q + "q.norm": (a.dim,),
                      q + "k.norm": (a.dim,), q + "g": (a.heads, d), q + "o": (d, a.heads * a.vdim)})
            q = p + "right."
            t.update({q + "q": (r.heads * r.dim, d), q + "k": (r.heads * r.dim, d), q + "v": (r.heads * r.vdim, d), q + "g": (r.heads * r.vdim, d),
                      q + "o": (d, r.heads * r.vdim), q + "norm": (r.vdim,), q + "a1": (None, d), q + "a2": (r.heads * r.dim, None),
                      q + "a2.b": (r.heads * r.dim,)})
        if L.ff is not None:
            p = f"l{i}.mlp."
            t.update({p + "gate": (L.ff, d), p + "up": (L.ff, d), p + "down": (d, L.ff)})
    t["final.norm"] = (d,)
    t["head"] = (hp.n_vocab, d)
    return t


def _concrete(hp: LugovikHParams) -> Dict[str, Tuple[int, ...]]:
    return {k: tuple(hp.random_rank if n is None else n for n in s) for k, s in tensor_table(hp).items()}


def _unused(hp: LugovikHParams, name: str) -> bool:
    """Norms of a feed-forward the layer does not have."""
    layer, _, k = name.partition(".")
    return k in ("norm2", "norm2b") and layer[1:].isdigit() and int(layer[1:]) < hp.n_layer and hp.layers[int(layer[1:])].ff is None


def iter_checkpoint(directory: str, hp: LugovikHParams) -> Iterator[Tuple[str, torch.Tensor]]:
    """(name, CPU tensor) of every tensor of the model from the folder's safetensors file(s); checks names and shapes."""
    return checked_tensors(directory, tensor_table(hp), lambda n: _unused(hp, n))


def iter_random(hp: LugovikHParams, seed: int = 0, dtype: torch.dtype = torch.float32, device="cpu") -> Iterator[Tuple[str, torch.Tensor]]:
    """Random weights: matrices N(0, 1 / fan-in), norms around one, decays of a few to a few hundred tokens; drawn on ``device``."""
    dev = torch.device(device)
    gen = torch.Generator(device=dev)
    for name, shape in _concrete(hp).items():
        gen.manual_seed(_stream_seed(seed, name, 0))
        leaf = name.rsplit(".", 1)[-1]
        std = 1.0 / hp.embed_scale if name == "embed" else 0.5 if leaf == "conv" else 0.2 if len(shape) == 1 else shape[1] ** -0.5
        x = torch.empty(shape, dtype=dtype, device=dev).normal_(0.0, std, generator=gen)
        yield name, x + 1 if "norm" in leaf else x - 3 if leaf == "dt_bias" else x


def load_config(directory: str) -> LugovikHParams:
    with open(os.path.join(directory, "config.json")) as f:
        return LugovikHParams.from_config(json.load(f))


class _Layer:
    __slots__ = ("norm1", "norm1b", "norm2", "norm2b", "w_in", "w_low", "w_o", "w_gate", "w_up", "w_down", "mix", "attn", "cols", "low_cols", "rope")

    def __init__(self):
        for s in self.__slots__:
            setattr(self, s, None)


# ---- model -----------------------------------------------------------------------------------------------------------------------
class LugovikModel:
    recurrent = True                  # sequences carry a state besides their cached rows (see Scheduler.set_recurrent)
    split = False
    comm = None

    def __init__(self, hp: LugovikHParams, weights: Iterable[Tuple[str, torch.Tensor]], dtype: torch.dtype = torch.bfloat16, device="cpu",
                 max_positions: int = 8192, block_size: int = 64):
        self.hp, self.dtype, self.device = hp, dtype, torch.device(device)
        self.spec = ShardSpec()
        self.block_size, self.max_positions = block_size, max_positions
        self.tensor_hook = None       # called as tensor_hook(name, tensor) with every layer's residual; steps then run eagerly
        self.layers = [_Layer() for _ in hp.layers]
        tables: Dict[Rotation, torch.Tensor] = {}
        for L, s in zip(self.layers, hp.layers):
            if isinstance(s.mixer, ParallelMixer):
                rot = s.mixer.left.rot
                if rot not in tables:
                    tables[rot] = rope_table(max_positions, rot, self.device)
                L.rope = tables[rot]
        self._load(weights)

    # ---- weight intake ---------------------------------------------------------------------------------------------------------
    def _load(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> None:
        hp, dev, f32 = self.hp, self.device, torch.float32
        table = tensor_table(hp)
        pend: Dict[str, torch.Tensor] = {}
        todo = [set(k for k in table if k.startswith(f"l{i}.")) for i in range(hp.n_layer)]
        seen = set()
        for name, t in weights:
            _trace.log_tensor(name, t.shape, t.dtype, "")
            if name not in table:
                if _unused(hp, name):
                    continue
                raise KeyError(f"unknown tensor {name}")
            if not fits(t.shape, table[name]):
                raise ValueError(f"{name}: shape {tuple(t.shape)} != expected {table[name]}")
            seen.add(name)
            small = t.dim() == 1 or name.endswith(".conv")
            pend[name] = t.to(device=dev, dtype=f32 if small else self.dtype).contiguous()
            li = name.split(".", 1)[0]
            if li[0] == "l" and li[1:].isdigit():
                i = int(li[1:])
                todo[i].discard(name)
                if not todo[i]:                               # complete: stack it and let the parts go
                    self._finish_layer(i, pend)
        missing = [n for n in table if n not in seen]
        if missing:
            raise ValueError(f"missing tensors: {len(missing)}, e.g. {missing[:3]}")
        self.embed, self.final_norm, self.head = pend.pop("embed"), pend.pop("final.norm"), pend.pop("head")

    def _finish_layer(self, i: int, pend: Dict[str, torch.Tensor]) -> None:
        L, s, eps = self.layers[i], self.hp.layers[i], self.hp.eps
        take = lambda k: pend.pop(f"l{i}.{k}")                                  # noqa: E731
        m = s.mixer
        L.norm1, L.norm1b = take("norm1"), take("norm1b")
        if s.ff is not None:
            L.norm2, L.norm2b = take("norm2"), take("norm2b")
            L.w_gate, L.w_up, L.w_down = take("mlp.gate"), take("mlp.up"), take("mlp.down")
        if isinstance(m, Mamba2Mixer):
            gn = m.groups * m.state
            w = take("mix.in")
            L.w_in, c = stack_rows([("z", w[:m.inner]), ("x", w[m.inner:2 * m.inner + 2 * gn]), ("dt", w[2 * m.inner + 2 * gn:])])
            L.w_o = take("mix.o")
            L.mix = StateMix("ssd", m.heads, m.state, m.vdim, m.heads // m.groups, q_off=c["x"] + m.inner + gn, k_off=c["x"] + m.inner,
                             v_off=c["x"], s_off=c["dt"], taps=m.conv, conv0=c["x"], conv_w=take("mix.conv").t().contiguous(),
                             conv_b=take("mix.conv.b"), bias=take("mix.dt_bias"), neg_a=-torch.exp(take("mix.A_log")), skip=take("mix.D"),
                             norm_w=take("mix.norm"), norm_groups=m.norm_groups, eps=eps)
        elif isinstance(m, DeltaMixer):
            a1, a2, g1, g2 = take("mix.a1"), take("mix.a2"), take("mix.g1"), take("mix.g2")
            self._check_rank(i, "a", a1, a2)
            self._check_rank(i, "g", g1, g2)
            L.w_in, c = stack_rows([(k, take("mix." + k)) for k in ("q", "k", "v", "b")] + [("a1", a1), ("g1", g1)])
            conv, _ = stack_rows([(k, take(f"mix.{k}.conv")) for k in ("q", "k", "v")])
            L.w_low, rows = block_diagonal([a2, g2])
            L.low_cols, L.w_o = rows, take("mix.o")
            L.mix = StateMix("delta", m.heads, m.dim, m.vdim, m.heads // m.kv_heads, q_off=c["q"], k_off=c["k"], v_off=c["v"], s_off=c["b"],
                             taps=m.conv, conv0=c["q"], conv_w=conv.t().contiguous(), bias=take("mix.dt_bias"), neg_a=-torch.exp(take("mix.A_log")),
                             norm_w=take("mix.norm"), q_scale=m.dim ** -0.5, eps=eps)
        else:
            a, r = m.left, m.right
            a1, a2 = take("mix.right.a1"), take("mix.right.a2")
            self._check_rank(i, "right.a", a1, a2)
            L.w_in, c = stack_rows([("l" + k, take("mix.left." + k)) for k in ("q", "k", "v", "g")] +
                                   [("r" + k, take("mix.right." + k)) for k in ("q", "k", "v", "g")] + [("a1", a1)])
            L.w_low, _ = block_diagonal([a2])
            wl, wr = take("mix.left.o"), take("mix.right.o")
            nl = up(wl.shape[1])                             # the right half's first column
            L.w_o = torch.zeros(wl.shape[0], nl + wr.shape[1], dtype=wl.dtype, device=wl.device)
            L.w_o[:, :wl.shape[1]], L.w_o[:, nl:] = wl, wr
            c["y"] = nl
            L.attn = Gqa(a.heads, a.kv_heads, a.dim, a.vdim, a.rot.dims, a.scale, take("mix.left.q.norm"), take("mix.left.k.norm"), a.softcap,
                         chunk=a.chunk, sink=True, eps=eps, out_scale=m.left_scale)
            L.mix = StateMix("linear", r.heads, r.dim, r.vdim, q_off=c["rq"], k_off=c["rk"], v_off=c["rv"], bias=take("mix.right.a2.b"),
                             norm_w=take("mix.right.norm"), q_scale=r.dim ** -0.5, inv_tau=1.0 / r.tau, eps=eps, out_scale=m.right_scale)
        L.cols = c

    @staticmethod
    def _check_rank(i: int, name: str, w1: torch.Tensor, w2: torch.Tensor) -> None:
        if w1.shape[0] != w2.shape[1]:
            raise ValueError(f"layer {i}: the low-rank projection {name} has inner widths {w1.shape[0]} and {w2.shape[1]}")

    def weight_bytes(self) -> int:
        ts = [self.embed, self.final_norm, self.head]
        for L in self.layers:
            ts += [getattr(L, k) for k in L.__slots__] + [v for x in (L.mix, L.attn) if x is not None for v in vars(x).values()]
        return sum(t.numel() * t.element_size() for t in ts if isinstance(t, torch.Tensor))

    # ---- cache -------------------------------------------------------------------------------------------------------------------
    def cache_bytes_per_token(self) -> int:
        el = torch.empty(0, dtype=self.dtype).element_size()
        return sum(L.attn.kv_row * el for L in self.layers if L.attn is not None)

    def make_cache(self, n_slots: int, n_seqs: int):
        """Paged rows of ``n_slots`` tokens for the attention, a state row per sequence slot for the recurrences and convolutions."""
        from ..runtime.cache import HybridCache
        state = {"conv": [(tuple([L.mix.taps, L.mix.conv_w.shape[1]]), self.dtype) if L.mix.taps else None for L in self.layers],
                 "mix": [((L.mix.heads, L.mix.dim, L.mix.vdim), torch.float32) for L in self.layers]}
        return HybridCache([L.attn.kv_row if L.attn is not None else None for L in self.layers], state, n_slots, n_seqs, self.dtype, self.device,
                           self.block_size)

    # ---- forward -----------------------------------------------------------------------------------------------------------------
    def _mix(self, i: int, L: _Layer, m: Any, h: torch.Tensor, b: ForwardBatch, cache, single: bool) -> torch.Tensor:
        T, c, n = h.shape[0], L.cols, L.mix.heads * L.mix.vdim
        proj = ops.linear(h, L.w_in)
        y0, dec, gate = 0, None, None
        if L.w_low is not None:
            a0 = c["a1"]
            low = ops.linear(proj[:, a0:a0 + L.w_low.shape[1]], L.w_low)
            dec = low[:, :L.mix.heads * L.mix.dim]
        if isinstance(m, Mamba2Mixer):
            gate = proj[:, c["z"]:c["z"] + n]
        elif isinstance(m, DeltaMixer):
            gate = low[:, L.low_cols[1]:L.low_cols[1] + n]
        else:
            a, y0 = L.attn, c["y"]
            gate = proj[:, c["rg"]:c["rg"] + n]
        make = torch.zeros if y0 > (L.attn.heads * L.attn.vdim if L.attn is not None else 0) else torch.empty     # columns nobody writes
        y = make(T, y0 + n, dtype=h.dtype, device=h.device)
        if L.attn is not None:
            q = ops.gqa_qkv_post(a, proj[:, c["lq"]:c["lq"] + a.heads * a.dim], proj[:, c["lk"]:c["lk"] + a.kv_heads * a.dim],
                                 proj[:, c["lv"]:c["lv"] + a.kv_heads * a.vdim], L.rope, b.positions, b.slot_mapping, cache[i])
            ops.gqa_attention(a, q, cache[i], proj[:, c["lg"]:c["lg"] + a.heads], b.block_tables, b.seq_lens, b.q_start, self.block_size,
                              b.max_q_len, b.attn_meta, y[:, :y0])
        ops.state_mix(L.mix, proj, dec, gate, cache.state["conv"][i], cache.state["mix"][i], b.seq_slots, b.positions, b.q_start, single, y[:, y0:])
        return ops.linear(y, L.w_o)

    @torch.no_grad()
    def forward(self, batch: ForwardBatch, cache) -> torch.Tensor:
        """fp32 logits [len(out_rows), n_vocab]; ``cache`` is a ``HybridCache`` of this model."""
        hp, b = self.hp, batch
        single = b.max_q_len == 1 and b.seq_lens.shape[0] == b.tokens.shape[0]       # row t is sequence t's only token
        norms = [L.norm1 for L in self.layers] + [None]

        def nxt(w):                   # the norm that follows a residual update
            return None if w is None else (w, hp.eps, None)

        x, h, _ = ops.embed_norm(self.embed, b.tokens, None, hp.eps, nxt(norms[0]), hp.embed_scale)
        for i, (L, s) in enumerate(zip(self.layers, hp.layers)):
            o = self._mix(i, L, s.mixer, h, b, cache, single)
            x, h = ops.post_norm(x, o, L.norm1b, hp.eps, nxt(L.norm2 if s.ff is not None else norms[i + 1]))
            if s.ff is not None:
                f = ops.linear(ops.gateup(h, L.w_gate, L.w_up, "gelu_tanh"), L.w_down)
                x, h = ops.post_norm(x, f, L.norm2b, hp.eps, nxt(norms[i + 1]))
            if self.tensor_hook is not None:
                self.tensor_hook(f"blk.{i}.mix_out", o)
                self.tensor_hook(f"blk.{i}.ffn_out", x.clone())
        if b.out_rows.shape[0] == 0:
            return torch.empty(0, hp.n_vocab, dtype=torch.float32, device=self.device)
        xo = ops.rms_rows(x, b.out_rows, self.final_norm, hp.eps, self.dtype)
        logits = ops.linear(xo, self.head, out_dtype=torch.float32)
        if self.tensor_hook is not None:
            self.tensor_hook("result_norm", xo)
            self.tensor_hook("result_output", logits)
        return logits
