"""Zomavik: a decoder whose layers run attention beside a selective scan, next to a feed-forward; some layers run several times.

A layer adds two scaled sublayers of one fp32 residual row, each behind a norm of its own:
``x <- x + ls1 * mixer(norm1(x)) + ls2 * ff(norm2(x))`` (a layer may have no feed-forward).  What the layers are made of:

* **mixer** -- grouped-query attention (biases on q, k and v, rotate-half RoPE on a part of the head, softcap, a learned sink per head) and
  a selective scan (short convolution, step sizes through a low-rank projection, one decay per channel and state) on one input,
  their weighted outputs added;
* **feed-forward** -- dense with a squared relu, or experts: softmax scores, only experts of the best groups, weights scaled to sum
  to one, a shared expert behind a gate of its own;
* **loop** -- layers ``start`` to ``stop`` run ``times`` times with the same weights; every pass begins with ``x <- W [x; x0]``, x0 the
  embedding output, and has cache rows and states of its own.

Attention rows are paged; scan states and the convolutions' last inputs live in one row per sequence slot and layer run
(``runtime/cache.py:HybridCache``), and a batch range that starts at position 0 starts from zeros.

Channels and states of the scan are padded to multiples of 8 with zero weights.  One product of ``norm1(x)`` feeds q, k, v and both halves
of the scan (the biases are its epilogue), one product of the halves' results side by side is the mixer's output.  A pass' ``W x0`` is
the same in every pass and computed once.  The shared expert joins the grouped expert products when its width is a multiple of
theirs.  On a GPU a decode step runs per layer: input GEMM, rotation, attention, convolution, two GEMMs and the scan step,
output GEMM, router, gating, expert sort, two grouped GEMMs, and one ``scaled_update`` launch for the combine, both scales, the residual
and the next layer's two norms.  ``dtype`` float32 runs the same graph with fp32 kernels.
"""
from __future__ import annotations

import json
import math
import os
from dataclasses import dataclass, field
from typing import Any, Dict, Iterable, Iterator, List, Optional, Tuple

import torch

from .. import ops
from ..ops.specs import Gqa, RowNorms, SelectiveScan
from ..utils import trace as _trace
from .deepseek2 import ForwardBatch
from .folder import Rotation, checked_tensors, fits, rope_table, stack_rows, up
from .weights import ShardSpec, _stream_seed

ARCH = "Zomavik"
MAX_EXPERTS, MAX_CHOICES, MAX_STATE = 256, 32, 256           # what the routing and scan kernels are built for


# ---- configuration -----------------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class AttentionPart:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float                 # 0: none
    rot: Rotation


@dataclass(frozen=True)
class ScanPart:
    inner: int
    state: int
    dt_rank: int
    conv: int


@dataclass(frozen=True)
class ParallelMixer:
    left: AttentionPart
    right: ScanPart
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class Dense:
    ff: int


@dataclass(frozen=True)
class Experts:
    ff: int
    experts: int
    top: int
    groups: int = 1
    keep: int = 1
    shared: Optional[int] = None   # width of the shared expert


@dataclass(frozen=True)
class LayerSpec:
    mixer: ParallelMixer
    mlp: Any                       # Dense | Experts | None


@dataclass(frozen=True)
class Loop:
    start: int
    stop: int
    times: int


def _mixer(kind: str, m: Dict[str, Any]) -> ParallelMixer:
    if kind != "parallel":
        raise ValueError(f"unknown mixer {kind!r}")
    a, r = m["left"], m["right"]
    left = AttentionPart(int(a["heads"]), int(a["kv_heads"]), int(a["dim"]), int(a["vdim"]), float(a["scale"]), float(a.get("softcap") or 0.0),
                         Rotation(int(a["rot"]["dims"]), float(a["rot"]["base"])))
    if left.heads % left.kv_heads or left.rot.dims % 2 or left.rot.dims > left.dim:
        raise ValueError("heads must be a multiple of kv_heads, the rotated dimensions an even part of the head")
    right = ScanPart(int(r["inner"]), int(r["state"]), int(r["dt_rank"]), int(r["conv"]))
    if right.conv < 1 or not 1 <= right.state <= MAX_STATE:
        raise ValueError(f"a convolution has at least one tap, a channel 1 to {MAX_STATE} states")
    return ParallelMixer(left, right, float(m["left_scale"]), float(m["right_scale"]))


def _mlp(m: Optional[Dict[str, Any]]):
    if m is None:
        return None
    if m.get("kind") == "dense":
        return Dense(int(m["ff"]))
    if m.get("kind") != "moe":
        raise ValueError(f"unknown feed-forward {m.get('kind')!r}")
    r, sh = m["router"], m.get("shared")
    g = r.get("groups") or {"count": 1, "keep": 1}
    x = Experts(int(m["expert"]["ff"]), int(r["experts"]), int(r["top"]), int(g["count"]), int(g["keep"]), None if sh is None else int(sh["ff"]))
    if not 1 <= x.experts <= MAX_EXPERTS or not 1 <= x.top <= MAX_CHOICES:
        raise ValueError(f"top {x.top} of {x.experts} experts: at most {MAX_CHOICES} of {MAX_EXPERTS}")
    if x.experts % x.groups or not 1 <= x.keep <= x.groups <= 32 or x.top > x.experts // x.groups * x.keep:
        raise ValueError(f"top {x.top} of the best {x.keep} of {x.groups} groups of {x.experts} experts")
    return x


@dataclass
class ZomavikHParams:
    n_vocab: int
    n_embd: int
    eps: float
    embed_scale: float
    logit_scale: float = 1.0
    logit_softcap: float = 0.0     # 0: none
    layers: List[LayerSpec] = field(default_factory=list)
    loop: Optional[Loop] = None
    bos_id: int = -1               # token ids only: the design names no special tokens
    eos_id: int = -1
    n_ctx_train: int = 1 << 20

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @property
    def runs(self) -> List[int]:
        """The layers in the order they run."""
        n, p = self.n_layer, self.loop
        return list(range(n)) if p is None else [*range(p.start), *(list(range(p.start, p.stop)) * p.times), *range(p.stop, n)]

    @property
    def passes(self) -> List[int]:
        """Places in ``runs`` where a pass of the loop begins."""
        p = self.loop
        return [] if p is None else [p.start + k * (p.stop - p.start) for k in range(p.times)]

    @classmethod
    def from_config(cls, cfg: Dict[str, Any]) -> "ZomavikHParams":
        if cfg.get("architecture") != ARCH:
            raise ValueError(f"architecture {cfg.get('architecture')!r} is not {ARCH}")
        layers: List[LayerSpec] = []
        for i, e in enumerate(cfg["layers"]):
            try:
                layers.append(LayerSpec(_mixer(e["type"], e["mixer"]), _mlp(e.get("mlp"))))
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
        lp = cfg.get("loop")
        if lp is not None:
            lp = Loop(int(lp["start"]), int(lp["stop"]), int(lp["times"]))
            if not 0 <= lp.start < lp.stop <= len(layers) or lp.times < 1:
                raise ValueError(f"loop {lp} over {len(layers)} layers")
        scale = cfg.get("logit_scale")
        return cls(n_vocab=int(cfg["vocab"]), n_embd=int(cfg["width"]), eps=float(cfg["norm"]["eps"]), embed_scale=float(cfg["embedding"]["scale"]),
                   logit_scale=1.0 if scale is None else float(scale), logit_softcap=float(cfg.get("logit_softcap") or 0.0), layers=layers, loop=lp)

    def to_config(self) -> Dict[str, Any]:
        out = []
        for L in self.layers:
            a, r, m = L.mixer.left, L.mixer.right, L.mlp
            left = dict(heads=a.heads, kv_heads=a.kv_heads, dim=a.dim, vdim=a.vdim, scale=a.scale, softcap=a.softcap, rot=dict(base=a.rot.base, dims=a.rot.dims))
            mix = dict(left=left, left_scale=L.mixer.left_scale, right=dict(inner=r.inner, state=r.state, dt_rank=r.dt_rank, conv=r.conv),
                       right_scale=L.mixer.right_scale)
            mlp = m
            if isinstance(m, Dense):
                mlp = dict(kind="dense", ff=m.ff)
            elif m is not None:
                mlp = dict(kind="moe", expert=dict(ff=m.ff), router=dict(experts=m.experts, top=m.top, groups=dict(count=m.groups, keep=m.keep)))
                if m.shared is not None:
                    mlp["shared"] = dict(ff=m.shared)
            out.append(dict(type="parallel", mixer=mix, mlp=mlp))
        cfg = dict(architecture=ARCH, vocab=self.n_vocab, width=self.n_embd, norm=dict(eps=self.eps), embedding=dict(scale=self.embed_scale),
                   logit_scale=self.logit_scale, logit_softcap=self.logit_softcap, layers=out)
        if self.loop is not None:
            cfg["loop"] = dict(start=self.loop.start, stop=self.loop.stop, times=self.loop.times)
        return cfg

    def n_params(self) -> int:
        return sum(math.prod(s) for s in tensor_table(self).values())


def preset(name: str) -> ZomavikHParams:
    """Named shapes for tests, examples and benchmarks (random weights)."""
    name = name.lower().replace("_", "-")

    def stack(n, dense, mixer, experts, dense_ff):
        return [LayerSpec(mixer, Dense(dense_ff) if i < dense else experts) for i in range(n)]
    if name == "zomavik-tiny":
        mix = ParallelMixer(AttentionPart(4, 2, 40, 24, 0.2, 12.0, Rotation(24, 10000.0)), ScanPart(112, 12, 10, 4), 0.8, 0.7)
        return ZomavikHParams(n_vocab=600, n_embd=160, eps=1e-5, embed_scale=2.0, logit_scale=0.8, logit_softcap=20.0,
                              layers=stack(4, 1, mix, Experts(64, 12, 3, 3, 2, 64), 224), loop=Loop(1, 3, 2))
    if name in ("zomavik-lite", "zomavik-v2"):
        # the layer sizes of DeepSeek-V2-Lite (64 experts of which 6 run) and DeepSeek-V2 (160 experts in 8 groups), two shared experts' width
        w, h, n, experts, loop = (2048, 16, 10, Experts(1408, 64, 6, shared=2816), Loop(4, 6, 2)) if name == "zomavik-lite" else \
            (5120, 40, 3, Experts(1536, 160, 6, 8, 3, 3072), Loop(1, 2, 2))
        mix = ParallelMixer(AttentionPart(h, h // 4, 128, 128, 128 ** -0.5, 30.0, Rotation(128, 500000.0)), ScanPart(2 * w, 16, w // 16, 4), 0.7, 0.7)
        return ZomavikHParams(n_vocab=102400, n_embd=w, eps=1e-6, embed_scale=1.0, logit_scale=1.0, logit_softcap=30.0,
                              layers=stack(n, 0, mix, experts, 0), loop=loop)
    raise KeyError(name)


# ---- weights -------------------------------------------------------------------------------------------------------------------
def tensor_table(hp: ZomavikHParams) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint tensor name -> shape."""
    d = hp.n_embd
    t: Dict[str, Tuple[int, ...]] = {"embed": (hp.n_vocab, d)}
    if hp.loop is not None:
        t["loop.in"] = (d, 2 * d)
    for i, L in enumerate(hp.layers):
        p, a, r, m = f"l{i}.", L.mixer.left, L.mixer.right, L.mlp
        for k in ("norm1", "ls1") + (("norm2", "ls2") if m is not None else ()):
            t[p + k] = (d,)
        q = p + "mix.left."
        for k, n in (("q", a.heads * a.dim), ("k", a.kv_heads * a.dim), ("v", a.kv_heads * a.vdim)):
            t[q + k] = (n, d)
            t[q + k + ".b"] = (n,)
        t.update({q + "sink": (a.heads,), q + "o": (d, a.heads * a.vdim)})
        q = p + "mix.right."
        t.update({q + "in": (2 * r.inner, d), q + "conv": (r.inner, r.conv), q + "conv.b": (r.inner,), q + "x": (r.dt_rank + 2 * r.state, r.inner),
                  q + "dt": (r.inner, r.dt_rank), q + "dt.b": (r.inner,), q + "A_log": (r.inner, r.state), q + "D": (r.inner,), q + "o": (d, r.inner)})
        p += "mlp."
        if isinstance(m, Dense):
            t.update({p + "up": (m.ff, d), p + "down": (d, m.ff)})
        elif m is not None:
            for e, n in [(f"e{j}", m.ff) for j in range(m.experts)] + ([("shared", m.shared)] if m.shared is not None else []):
                t.update({p + e + ".gate": (n, d), p + e + ".up": (n, d), p + e + ".down": (d, n)})
            t[p + "router"] = (m.experts, d)
            if m.shared is not None:
                t[p + "shared.sg"] = (1, d)
    t["final.norm"] = (d,)
    t["head"] = (hp.n_vocab, d)
    return t


def _unused(hp: ZomavikHParams, name: str) -> bool:
    """Norm and scale of a feed-forward the layer does not have."""
    layer, _, k = name.partition(".")
    return k in ("norm2", "ls2") and layer[1:].isdigit() and int(layer[1:]) < hp.n_layer and hp.layers[int(layer[1:])].mlp is None


def iter_checkpoint(directory: str, hp: ZomavikHParams) -> Iterator[Tuple[str, torch.Tensor]]:
    """(name, CPU tensor) of every tensor of the model from the folder's safetensors file(s); checks names and shapes."""
    return checked_tensors(directory, tensor_table(hp), lambda n: _unused(hp, n))


def iter_random(hp: ZomavikHParams, seed: int = 0, dtype: torch.dtype = torch.float32, device="cpu") -> Iterator[Tuple[str, torch.Tensor]]:
    """Random weights: matrices N(0, 1 / fan-in), norms and layer scales around one, decays of a few to a few hundred tokens."""
    dev = torch.device(device)
    gen = torch.Generator(device=dev)
    for name, shape in tensor_table(hp).items():
        gen.manual_seed(_stream_seed(seed, name, 0))
        leaf = name.rsplit(".", 1)[-1]
        std = 1.0 if name == "embed" else 0.5 if leaf in ("conv", "A_log") else 0.2 if len(shape) == 1 else shape[1] ** -0.5
        x = torch.empty(shape, dtype=dtype, device=dev).normal_(0.0, std, generator=gen)
        yield name, x + 1 if "norm" in leaf or leaf in ("ls1", "ls2") else x - 3 if name.endswith("dt.b") else x


def load_config(directory: str) -> ZomavikHParams:
    with open(os.path.join(directory, "config.json")) as f:
        return ZomavikHParams.from_config(json.load(f))


def _padded(t: torch.Tensor, *shape: int) -> torch.Tensor:
    """``t`` in the corner of a zero tensor."""
    if tuple(t.shape) == shape:
        return t
    out = torch.zeros(shape, dtype=t.dtype, device=t.device)
    out[tuple(slice(0, n) for n in t.shape)] = t
    return out


class _Layer:
    __slots__ = ("norm1", "norm2", "ls1", "ls2", "w_in", "b_in", "cols", "w_o", "y_col", "attn", "rope", "scan", "conv_w", "conv_b", "w_x", "w_dt",
                 "w_up", "w_down", "router", "n_merged", "w_gate_exps", "w_up_exps", "w_down_exps", "w_gate_sh", "w_up_sh", "w_down_sh")

    def __init__(self):
        for s in self.__slots__:
            setattr(self, s, None)


# ---- model -----------------------------------------------------------------------------------------------------------------------
class ZomavikModel:
    recurrent = True                  # sequences carry a state besides their cached rows (see Scheduler.set_recurrent)
    split = False
    comm = None

    def __init__(self, hp: ZomavikHParams, weights: Iterable[Tuple[str, torch.Tensor]], dtype: torch.dtype = torch.bfloat16, device="cpu",
                 max_positions: int = 8192, block_size: int = 64):
        self.hp, self.dtype, self.device = hp, dtype, torch.device(device)
        self.spec = ShardSpec()
        self.block_size, self.max_positions = block_size, max_positions
        self.tensor_hook = None       # called as tensor_hook(name, tensor) with every layer run's residual; steps then run eagerly
        self.runs, self.passes = hp.runs, set(hp.passes)
        self.layers = [_Layer() for _ in hp.layers]
        tables: Dict[Rotation, torch.Tensor] = {}
        for L, s in zip(self.layers, hp.layers):
            rot = s.mixer.left.rot
            if rot not in tables:
                tables[rot] = rope_table(max_positions, rot, self.device)
            L.rope = tables[rot]
        self.loop_x = self.loop_x0 = None
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
            if i >= 0 and base.startswith("mlp.") and isinstance(hp.layers[i].mlp, Experts) and base.count(".") == 2 and base[-3:] != ".sg":
                self._take_expert(i, *base.split(".")[1:], t)          # straight into the stacked tensors: nothing is held twice
            else:
                small = t.dim() == 1 or base.endswith((".conv", ".A_log"))
                pend[name] = t.to(device=dev, dtype=f32 if small else self.dtype).contiguous()
            if i >= 0:
                todo[i].discard(name)
                if not todo[i]:                               # complete: stack it and let the parts go
                    self._finish_layer(i, pend)
        missing = [n for n in table if n not in seen]
        if missing:
            raise ValueError(f"missing tensors: {len(missing)}, e.g. {missing[:3]}")
        self.embed, self.final_norm, self.head = pend.pop("embed"), pend.pop("final.norm"), pend.pop("head")
        if hp.loop is not None:
            w = pend.pop("loop.in")
            self.loop_x, self.loop_x0 = w[:, :hp.n_embd].contiguous(), w[:, hp.n_embd:].contiguous()

    def _take_expert(self, i: int, who: str, kind: str, t: torch.Tensor) -> None:
        L, m, d = self.layers[i], self.hp.layers[i].mlp, self.hp.n_embd
        if L.n_merged is None:            # a shared expert as wide as n routed ones is a sum over n experts of that width
            n = m.shared // m.ff if m.shared is not None and m.shared % m.ff == 0 else 0
            L.n_merged = n if m.experts + n <= MAX_EXPERTS and m.top + n <= MAX_CHOICES else 0
            for k, s in (("gate", (m.ff, d)), ("up", (m.ff, d)), ("down", (d, m.ff))):
                setattr(L, f"w_{k}_exps", torch.empty((m.experts + L.n_merged,) + s, dtype=self.dtype, device=self.device))
        w = getattr(L, f"w_{kind}_exps")
        if who != "shared":
            w[int(who[1:])].copy_(t)
        elif L.n_merged:
            parts = t.reshape(L.n_merged, m.ff, d) if kind != "down" else t.reshape(d, L.n_merged, m.ff).transpose(0, 1)
            w[m.experts:].copy_(parts)
        else:
            setattr(L, f"w_{kind}_sh", t.to(device=self.device, dtype=self.dtype).contiguous())

    def _finish_layer(self, i: int, pend: Dict[str, torch.Tensor]) -> None:
        L, s = self.layers[i], self.hp.layers[i]
        take = lambda k: pend.pop(f"l{i}.{k}")                                  # noqa: E731
        a, r, m = s.mixer.left, s.mixer.right, s.mlp
        L.norm1, L.ls1 = take("norm1"), take("ls1")
        if m is not None:
            L.norm2, L.ls2 = take("norm2"), take("ls2")
        ch, N, R = up(r.inner), up(r.state), up(r.dt_rank)
        w = take("mix.right.in")
        L.w_in, c = stack_rows([(k, take("mix.left." + k)) for k in "qkv"] + [("x", w[:r.inner]), ("z", w[r.inner:])])
        L.b_in, L.cols = torch.zeros(L.w_in.shape[0], dtype=torch.float32, device=self.device), c
        for k in "qkv":
            b = take(f"mix.left.{k}.b")
            L.b_in[c[k]:c[k] + b.shape[0]] = b
        L.attn = Gqa(a.heads, a.kv_heads, a.dim, a.vdim, a.rot.dims, a.scale, softcap=a.softcap, sink=True, sink_w=take("mix.left.sink"),
                     out_scale=s.mixer.left_scale)
        L.conv_w, L.conv_b = _padded(take("mix.right.conv").t(), r.conv, ch).contiguous(), _padded(take("mix.right.conv.b"), ch)
        w, rows = take("mix.right.x"), (0, r.dt_rank, r.dt_rank + r.state, r.dt_rank + 2 * r.state)
        w, _ = stack_rows([(str(k), w[rows[k]:rows[k + 1]]) for k in range(3)])                      # dt | B | C
        L.w_x = _padded(w, w.shape[0], ch)
        L.w_dt = _padded(take("mix.right.dt"), ch, R)
        L.scan = SelectiveScan(ch, N, _padded(-torch.exp(take("mix.right.A_log")), ch, N), _padded(take("mix.right.D"), ch),
                               _padded(take("mix.right.dt.b"), ch), s.mixer.right_scale)
        wl, wr = take("mix.left.o"), take("mix.right.o")
        L.y_col = up(wl.shape[1])                             # the scan's first column
        L.w_o = torch.zeros(wl.shape[0], L.y_col + ch, dtype=wl.dtype, device=wl.device)
        L.w_o[:, :wl.shape[1]], L.w_o[:, L.y_col:L.y_col + r.inner] = wl, wr
        if isinstance(m, Dense):
            L.w_up, L.w_down = take("mlp.up"), take("mlp.down")
        elif m is not None:
            L.router = take("mlp.router")
            if m.shared is not None:
                L.router = torch.cat([L.router, take("mlp.shared.sg")], 0).contiguous()

    def weight_bytes(self) -> int:
        ts = [self.embed, self.final_norm, self.head, self.loop_x, self.loop_x0]
        for L in self.layers:
            ts += [getattr(L, k) for k in L.__slots__] + [v for x in (L.scan, L.attn) for v in vars(x).values()]
        return sum(t.numel() * t.element_size() for t in ts if isinstance(t, torch.Tensor))

    # ---- cache -------------------------------------------------------------------------------------------------------------------
    def cache_bytes_per_token(self) -> int:
        el = torch.empty(0, dtype=self.dtype).element_size()
        return sum(self.layers[i].attn.kv_row * el for i in self.runs)

    def make_cache(self, n_slots: int, n_seqs: int):
        """Per layer run: paged rows of ``n_slots`` tokens for the attention, a state row per sequence slot for scan and convolution."""
        from ..runtime.cache import HybridCache
        Ls = [self.layers[i] for i in self.runs]
        state = {"conv": [((L.conv_w.shape[0] - 1, L.scan.channels), self.dtype) for L in Ls],
                 "scan": [((L.scan.channels, L.scan.state), torch.float32) for L in Ls]}
        return HybridCache([L.attn.kv_row for L in Ls], state, n_slots, n_seqs, self.dtype, self.device, self.block_size)

    # ---- forward -----------------------------------------------------------------------------------------------------------------
    def _mix(self, r: int, L: _Layer, h: torch.Tensor, b: ForwardBatch, cache, single: bool) -> torch.Tensor:
        T, c, a, m = h.shape[0], L.cols, L.attn, L.scan
        proj = ops.linear(h, L.w_in, residual=L.b_in.expand(T, -1))
        x, z = proj[:, c["x"]:c["x"] + m.channels], proj[:, c["z"]:c["z"] + m.channels]
        n = a.heads * a.vdim
        y = (torch.zeros if L.y_col > n else torch.empty)(T, L.y_col + m.channels, dtype=h.dtype, device=h.device)
        q = ops.gqa_qkv_post(a, proj[:, c["q"]:c["q"] + a.heads * a.dim], proj[:, c["k"]:c["k"] + a.kv_heads * a.dim],
                             proj[:, c["v"]:c["v"] + a.kv_heads * a.vdim], L.rope, b.positions, b.slot_mapping, cache[r])
        ops.gqa_attention(a, q, cache[r], None, b.block_tables, b.seq_lens, b.q_start, self.block_size, b.max_q_len, b.attn_meta, y[:, :n])
        xc = ops.causal_conv(x, L.conv_w, cache.state["conv"][r], b.seq_slots, b.positions, b.q_start, L.conv_b)
        low = ops.linear(xc, L.w_x)                           # dt | B | C
        R = L.w_dt.shape[1]
        dt = ops.linear(low[:, :R], L.w_dt)
        ops.selective_scan(m, xc, z, low[:, R:], dt, cache.state["scan"][r], b.seq_slots, b.positions, b.q_start, single, y[:, L.y_col:])
        return ops.linear(y, L.w_o)

    def _ff(self, L: _Layer, m: Any, h: torch.Tensor) -> Dict[str, Any]:
        """The feed-forward's part of ``ops.scaled_update``'s arguments."""
        if isinstance(m, Dense):
            return {"dense": ops.linear(ops.linear(h, L.w_up, unary=("relu2",)), L.w_down)}
        route = ops.moe_gate(h, L.router, None, m.top, m.groups, m.keep, 1.0, True, False, L.n_merged, shared_gate=m.shared is not None)
        y, dest = ops.moe_routed(h, route[0], route[1], L.w_gate_exps, L.w_up_exps, L.w_down_exps)
        out: Dict[str, Any] = {"moe": (y, dest, route[1])}
        if m.shared is not None and not L.n_merged:
            out["dense"], out["dense_gate"] = ops.linear(ops.gateup(h, L.w_gate_sh, L.w_up_sh, "silu"), L.w_down_sh), route[2]
        return out

    @torch.no_grad()
    def forward(self, batch: ForwardBatch, cache) -> torch.Tensor:
        """fp32 logits [len(out_rows), n_vocab]; ``cache`` is a ``HybridCache`` of this model."""
        hp, b = self.hp, batch
        single = b.max_q_len == 1 and b.seq_lens.shape[0] == b.tokens.shape[0]       # row t is sequence t's only token

        def norms(r):
            L = self.layers[self.runs[r]]
            return RowNorms(hp.eps, L.norm1, L.norm2)

        def nxt(r):                   # what follows a residual update; ahead of a pass its product takes the row as it is
            return None if r == len(self.runs) else RowNorms() if r in self.passes else norms(r)

        x, h, h2 = ops.embed_norm(self.embed, b.tokens, None, hp.eps, nxt(0), hp.embed_scale)
        if hp.loop is not None:       # the embedding output's part of W [x; x0], the same for every pass
            x0 = h if 0 in self.passes else ops.embed_norm(self.embed, b.tokens, None, hp.eps, RowNorms(), hp.embed_scale)[1]
            from_x0 = ops.linear(x0, self.loop_x0, out_dtype=torch.float32)
        for r, i in enumerate(self.runs):
            L, m = self.layers[i], hp.layers[i].mlp
            if r in self.passes:
                x = ops.linear(h, self.loop_x, residual=from_x0, out_dtype=torch.float32)
                x, h, h2 = ops.scaled_update(x, None, None, nxt=norms(r), dtype=self.dtype)
            o = self._mix(r, L, h, b, cache, single)
            ff = self._ff(L, m, h2) if m is not None else {}
            x, h, h2 = ops.scaled_update(x, o, L.ls1, L.ls2, nxt=nxt(r + 1), **ff)
            if self.tensor_hook is not None:
                self.tensor_hook(f"blk.{r}.mix_out", o)
                self.tensor_hook(f"blk.{r}.ffn_out", x.clone())
        if b.out_rows.shape[0] == 0:
            return torch.empty(0, hp.n_vocab, dtype=torch.float32, device=self.device)
        xo = ops.rms_rows(x, b.out_rows, self.final_norm, hp.eps, self.dtype)
        logits = ops.linear(xo, self.head, out_dtype=torch.float32, unary=("cap", hp.logit_scale, hp.logit_softcap))
        if self.tensor_hook is not None:
            self.tensor_hook("result_norm", xo)
            self.tensor_hook("result_output", logits)
        return logits
