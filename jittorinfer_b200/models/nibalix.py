"""Nibalix: a decoder whose layers are windowed latent attention or a minGRU recurrence, side by side with a mixture of experts.

Every layer is  ``h = norm(x); x <- x + m (sigmoid(W1 h + b1) * mixer(h + conv(h)) + sigmoid(W2 h + b2) * experts(h))``  over an
fp32 residual stream ``x``.  What the layers are made of:

* **norm** -- RMS norm whose stored weight is the deviation from one (kept here as ``1 + w``);
* **input convolution** -- a short causal convolution over time on each channel, ahead of the mixer only;
* **latent attention** -- the weight-absorbed MLA form of ``deepseek2.py`` with a sliding window, rotate-half RoPE and a plain
  query projection; a layer may read the latent rows another layer has cached (``kv_from``) and then stores none of its own;
* **minGRU** -- a gated recurrence with an fp32 state per sequence;
* **experts** -- top-k router over biased logits, weights = softmax over the chosen logits.

The state that is not paged -- the convolution's last inputs in every layer, the recurrence's state -- lives in one row per
sequence slot (``runtime/cache.py:HybridCache``); a batch range that starts at position 0 starts from zeros.

On a GPU, decode steps run per layer: gates GEMM, input GEMM, mixer, output GEMM, router, two grouped expert GEMMs, and one
``block_update`` launch that combines the experts, gates both sublayers, updates the residual, applies the next layer's norm and
convolution and advances the convolution's state.  ``dtype`` float32 runs the same graph with fp32 kernels throughout.
"""
from __future__ import annotations

import json
import logging
import os
from dataclasses import dataclass, field
from typing import Any, Dict, Iterable, Iterator, List, Optional, Tuple

import torch

from .. import ops
from ..utils import trace as _trace
from .deepseek2 import ForwardBatch
from .weights import ShardSpec, _stream_seed

ARCH = "Nibalix"
log = logging.getLogger("jittorinfer_b200.models")


# ---- configuration -----------------------------------------------------------------------------------------------------------
@dataclass(frozen=True)
class LatentMixer:
    heads: int
    dim: int                       # unrotated query / key dimensions per head
    rot_dim: int                   # rotated ones
    vdim: int
    kv_rank: int
    scale: float
    window: int                    # position i sees j with 0 <= i - j < window
    rope_base: float
    kv_from: Optional[int] = None  # layer whose cached rows this layer reads

    @property
    def kv_row(self) -> int:
        return self.kv_rank + self.rot_dim


@dataclass(frozen=True)
class GruMixer:
    width: int


@dataclass(frozen=True)
class Experts:
    ff: int
    experts: int
    top: int


@dataclass(frozen=True)
class LayerSpec:
    mixer: Any                     # LatentMixer | GruMixer
    mlp: Optional[Experts]


@dataclass
class NibalixHParams:
    n_vocab: int
    n_embd: int
    eps: float
    residual_mult: float
    taps: int
    layers: List[LayerSpec] = field(default_factory=list)
    bos_id: int = -1               # token ids only: the design names no special tokens
    eos_id: int = -1
    n_ctx_train: int = 1 << 20

    @property
    def n_layer(self) -> int:
        return len(self.layers)

    @classmethod
    def from_config(cls, cfg: Dict[str, Any]) -> "NibalixHParams":
        if cfg.get("architecture") != ARCH:
            raise ValueError(f"architecture {cfg.get('architecture')!r} is not {ARCH}")
        layers: List[LayerSpec] = []
        for i, e in enumerate(cfg["layers"]):
            m = e["mixer"]
            if e["type"] == "latent_attention":
                rot = m["rot"]
                if int(rot["dims"]) != int(m["rot_dim"]) or int(m["rot_dim"]) % 2:
                    raise ValueError(f"layer {i}: the rotation must cover the (even) rotated part")
                src = m.get("kv_from")
                mix = LatentMixer(int(m["heads"]), int(m["dim"]), int(m["rot_dim"]), int(m["vdim"]), int(m["kv_rank"]), float(m["scale"]),
                                  int(m["mask"]["size"]), float(rot["base"]), None if src is None else int(src))
                if mix.window < 1:
                    raise ValueError(f"layer {i}: the window must hold at least the position itself")
                if src is not None:
                    o = layers[int(src)].mixer if 0 <= int(src) < i else None
                    if not isinstance(o, LatentMixer) or o.kv_from is not None:
                        raise ValueError(f"layer {i}: kv_from {src} names no earlier layer with latent rows of its own")
                    if (o.kv_rank, o.rot_dim, o.rope_base) != (mix.kv_rank, mix.rot_dim, mix.rope_base):
                        raise ValueError(f"layer {i}: kv_from {src} has other row widths or another rotation")
            elif e["type"] == "mingru":
                mix = GruMixer(int(m["width"]))
            else:
                raise ValueError(f"layer {i}: unknown mixer {e['type']!r}")
            mlp = e.get("mlp")
            if mlp is not None:
                if mlp.get("kind") != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {mlp.get('kind')!r}")
                mlp = Experts(int(mlp["expert"]["ff"]), int(mlp["router"]["experts"]), int(mlp["router"]["top"]))
                if not 1 <= mlp.top <= mlp.experts:
                    raise ValueError(f"layer {i}: top {mlp.top} of {mlp.experts} experts")
            layers.append(LayerSpec(mix, mlp))
        return cls(n_vocab=int(cfg["vocab"]), n_embd=int(cfg["width"]), eps=float(cfg["norm"]["eps"]),
                   residual_mult=float(cfg["residual_mult"]), taps=int(cfg["canon"]["taps"]), layers=layers)

    def to_config(self) -> Dict[str, Any]:
        out = []
        for L in self.layers:
            m = L.mixer
            if isinstance(m, LatentMixer):
                mix = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale,
                       "mask": {"size": m.window}, "rot": {"base": m.rope_base, "dims": m.rot_dim}}
                if m.kv_from is not None:
                    mix["kv_from"] = m.kv_from
            else:
                mix = {"width": m.width}
            mlp = None if L.mlp is None else {"kind": "moe", "expert": {"ff": L.mlp.ff}, "router": {"experts": L.mlp.experts, "top": L.mlp.top}}
            out.append({"type": "latent_attention" if isinstance(m, LatentMixer) else "mingru", "mixer": mix, "mlp": mlp})
        return {"architecture": ARCH, "vocab": self.n_vocab, "width": self.n_embd, "norm": {"eps": self.eps},
                "residual_mult": self.residual_mult, "canon": {"taps": self.taps}, "layers": out}

    def n_params(self) -> int:
        n = 0
        for s in tensor_table(self).values():
            k = 1
            for x in s:
                k *= x
            n += k
        return n


def preset(name: str) -> NibalixHParams:
    """Named shapes for tests, examples and benchmarks (random weights)."""
    name = name.lower().replace("_", "-")

    def stack(n, gru_width, heads, dim, rot, vdim, rank, window, base, experts):
        """Recurrence, attention, attention, attention on the rows of the second -- repeated."""
        lat = lambda src=None: LatentMixer(heads, dim, rot, vdim, rank, (dim + rot) ** -0.5, window, base, src)      # noqa: E731
        out = []
        for i in range(n):
            k = i % 4
            mix = GruMixer(gru_width) if k == 0 else lat(i - 1 if k == 3 else None)
            out.append(LayerSpec(mix, experts))
        return out
    if name == "nibalix-tiny":
        return NibalixHParams(n_vocab=640, n_embd=192, eps=1e-5, residual_mult=0.4, taps=4,
                              layers=stack(4, 160, 4, 48, 16, 40, 80, 70, 10000.0, Experts(64, 8, 2)))
    if name == "nibalix-lite":
        # the layer sizes of DeepSeek-V2-Lite: width 2048, 16 heads, latent rows of 512 + 64, 64 experts of which 6 run
        return NibalixHParams(n_vocab=102400, n_embd=2048, eps=1e-6, residual_mult=0.5, taps=4,
                              layers=stack(12, 2048, 16, 128, 64, 128, 512, 512, 10000.0, Experts(1408, 64, 6)))
    if name == "nibalix-v2":
        # the layer sizes of DeepSeek-V2: width 5120, 128 heads, 160 experts of which 6 run
        return NibalixHParams(n_vocab=102400, n_embd=5120, eps=1e-6, residual_mult=0.5, taps=4,
                              layers=stack(4, 5120, 128, 128, 64, 128, 512, 1024, 10000.0, Experts(1536, 160, 6)))
    raise KeyError(name)


# ---- weights -------------------------------------------------------------------------------------------------------------------
def tensor_table(hp: NibalixHParams) -> Dict[str, Tuple[int, ...]]:
    """Checkpoint tensor name -> shape."""
    d = hp.n_embd
    t: Dict[str, Tuple[int, ...]] = {"embed": (hp.n_vocab, d), "embed.norm": (d,)}
    for i, L in enumerate(hp.layers):
        p, m = f"l{i}.", L.mixer
        t[p + "norm1"] = (d,)
        if isinstance(m, LatentMixer):
            t[p + "mix.q"] = (m.heads * (m.dim + m.rot_dim), d)
            if m.kv_from is None:
                t[p + "mix.dkv"] = (m.kv_row, d)
                t[p + "mix.dkv.norm"] = (m.kv_rank,)
            t[p + "mix.uk"] = (m.heads * m.dim, m.kv_rank)
            t[p + "mix.uv"] = (m.heads * m.vdim, m.kv_rank)
            t[p + "mix.o"] = (d, m.heads * m.vdim)
        else:
            for k in ("z", "x"):
                t[p + f"mix.{k}"] = (m.width, d)
                t[p + f"mix.{k}.b"] = (m.width,)
            t[p + "mix.g"] = (m.width, d)
            t[p + "mix.o"] = (d, m.width)
        if L.mlp is not None:
            for e in range(L.mlp.experts):
                t[p + f"mlp.e{e}.gate"] = (L.mlp.ff, d)
                t[p + f"mlp.e{e}.up"] = (L.mlp.ff, d)
                t[p + f"mlp.e{e}.down"] = (d, L.mlp.ff)
            t[p + "mlp.router"] = (L.mlp.experts, d)
            t[p + "mlp.router.b"] = (L.mlp.experts,)
        t[p + "canon1"] = (d, hp.taps)
        for k in ("rg1", "rg2") if L.mlp is not None else ("rg1",):
            t[p + k] = (d, d)
            t[p + k + ".b"] = (d,)
    t["final.norm"] = (d,)
    t["head"] = (hp.n_vocab, d)
    return t


def iter_checkpoint(directory: str, hp: NibalixHParams) -> Iterator[Tuple[str, torch.Tensor]]:
    """(name, CPU tensor) of every tensor of the model from the folder's safetensors file(s); checks names and shapes."""
    from ..gguf.convert_hf import Checkpoint
    ck = Checkpoint(directory)
    try:
        table = tensor_table(hp)
        have = set(ck.names())
        missing = [n for n in table if n not in have]
        if missing:
            raise KeyError(f"checkpoint is missing {len(missing)} tensors, e.g. {missing[:3]}")
        extra = sorted(have - set(table))
        if extra:
            raise ValueError(f"checkpoint has {len(extra)} tensors the model does not use, e.g. {extra[:3]}")
        for name, shape in table.items():
            t = ck.get(name)
            if tuple(t.shape) != tuple(shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)} != expected {shape}")
            yield name, t
    finally:
        ck.close()


def iter_random(hp: NibalixHParams, seed: int = 0, dtype: torch.dtype = torch.float32, device="cpu") -> Iterator[Tuple[str, torch.Tensor]]:
    """Random weights: matrices N(0, 1 / fan-in), norm deviations and biases small; drawn on ``device``."""
    dev = torch.device(device)
    gen = torch.Generator(device=dev)
    for name, shape in tensor_table(hp).items():
        gen.manual_seed(_stream_seed(seed, name, 0))
        std = 1.0 if name == "embed" else 0.2 if len(shape) == 1 else shape[1] ** -0.5
        x = torch.empty(shape, dtype=dtype, device=dev).normal_(0.0, std, generator=gen)
        yield name, x + 1 if name.endswith("dkv.norm") else x


def load_config(directory: str) -> NibalixHParams:
    with open(os.path.join(directory, "config.json")) as f:
        return NibalixHParams.from_config(json.load(f))


class _Layer:
    __slots__ = ("norm", "conv", "w_gates", "b1", "b2", "w_in", "w_o", "kv_norm", "w_uk", "w_uv", "w_kv_b", "zb", "xb", "router", "router_b",
                 "w_gate_exps", "w_up_exps", "w_down_exps")

    def __init__(self):
        for s in self.__slots__:
            setattr(self, s, None)


# ---- model -----------------------------------------------------------------------------------------------------------------------
class NibalixModel:
    recurrent = True                  # sequences carry a state besides their cached rows (see Scheduler.set_recurrent)
    split = False
    comm = None

    def __init__(self, hp: NibalixHParams, weights: Iterable[Tuple[str, torch.Tensor]], dtype: torch.dtype = torch.bfloat16, device="cpu",
                 max_positions: int = 8192, block_size: int = 64):
        self.hp, self.dtype, self.device = hp, dtype, torch.device(device)
        self.spec = ShardSpec()
        self.block_size, self.max_positions = block_size, max_positions
        if hp.n_embd % 8:
            raise ValueError("the model width must be a multiple of 8")
        self.tensor_hook = None       # called as tensor_hook(name, tensor) with every layer's residual; steps then run eagerly
        self.layers = [_Layer() for _ in hp.layers]
        self._load(weights)
        self.rope: Dict[Tuple[int, float], torch.Tensor] = {}
        for L in hp.layers:
            if isinstance(L.mixer, LatentMixer) and (L.mixer.rot_dim, L.mixer.rope_base) not in self.rope:
                self.rope[(L.mixer.rot_dim, L.mixer.rope_base)] = ops.ref.yarn_table(
                    max_positions, L.mixer.rot_dim, L.mixer.rope_base, 1.0, 0.0, 1.0, 0.0, 0.0, device=self.device)

    # ---- weight intake ---------------------------------------------------------------------------------------------------------
    def _load(self, weights: Iterable[Tuple[str, torch.Tensor]]) -> None:
        hp, dev, f32 = self.hp, self.device, torch.float32
        mat = lambda t: t.to(device=dev, dtype=self.dtype).contiguous()            # noqa: E731
        vec = lambda t: t.to(device=dev, dtype=f32).contiguous()                   # noqa: E731
        pend: Dict[str, torch.Tensor] = {}
        table, seen = tensor_table(hp), set()
        for name, t in weights:
            _trace.log_tensor(name, t.shape, t.dtype, "")
            if name not in table:
                raise KeyError(f"unknown tensor {name}")
            if tuple(t.shape) != tuple(table[name]):
                raise ValueError(f"{name}: shape {tuple(t.shape)} != expected {table[name]}")
            seen.add(name)
            if name == "embed":
                self.embed = mat(t)
            elif name == "embed.norm":
                self.embed_norm = 1 + vec(t)
            elif name == "final.norm":
                self.final_norm = 1 + vec(t)
            elif name == "head":
                self.head = mat(t)
            else:
                li, base = name.split(".", 1)
                i = int(li[1:])
                if base.startswith("mlp.e"):
                    # straight into the stacked expert tensors: nothing is held twice
                    L, E = self.layers[i], hp.layers[i].mlp
                    e, kind = base[5:].split(".")
                    slot = {"gate": "w_gate_exps", "up": "w_up_exps", "down": "w_down_exps"}[kind]
                    if getattr(L, slot) is None:
                        setattr(L, slot, torch.empty((E.experts,) + tuple(t.shape), dtype=self.dtype, device=dev))
                    getattr(L, slot)[int(e)].copy_(t)
                else:
                    pend[name] = vec(t) if t.dim() == 1 or base in ("canon1", "mlp.router") else mat(t)
        missing = [n for n in table if n not in seen]
        if missing:
            raise ValueError(f"missing tensors: {len(missing)}, e.g. {missing[:3]}")
        for i, (L, s) in enumerate(zip(self.layers, hp.layers)):
            take = lambda k: pend.pop(f"l{i}.{k}")                                  # noqa: B023,E731
            m = s.mixer
            L.norm = 1 + take("norm1")
            L.conv = take("canon1").t().contiguous()                                # [taps, width]
            L.w_gates, L.b1 = take("rg1"), take("rg1.b")
            if s.mlp is not None:
                L.w_gates, L.b2 = torch.cat([L.w_gates, take("rg2")], 0), take("rg2.b")
                L.router, L.router_b = take("mlp.router"), take("mlp.router.b")
            if isinstance(m, LatentMixer):
                L.w_in = take("mix.q")
                if m.kv_from is None:
                    L.w_in, L.kv_norm = torch.cat([L.w_in, take("mix.dkv")], 0), take("mix.dkv.norm")
                uk = take("mix.uk").view(m.heads, m.dim, m.kv_rank)
                L.w_uv = take("mix.uv").view(m.heads, m.vdim, m.kv_rank)
                L.w_uk = uk.transpose(1, 2).contiguous()                            # [H, r, dn]: q_abs = q_nope @ w_uk[h]^T
                if self.dtype == torch.bfloat16 and (m.dim, m.rot_dim, m.vdim, m.kv_rank) == (128, 64, 128, 512):
                    # prompt portions expand k | v per head from the cached rows (the shape the prompt kernel is built for)
                    L.w_kv_b = torch.cat([uk, L.w_uv], 1).reshape(m.heads * (m.dim + m.vdim), m.kv_rank)
            else:
                L.w_in = torch.cat([take("mix.z"), take("mix.x"), take("mix.g")], 0)
                L.zb, L.xb = take("mix.z.b"), take("mix.x.b")
            L.w_o = take("mix.o")

    def weight_bytes(self) -> int:
        ts = [self.embed, self.embed_norm, self.final_norm, self.head] + [getattr(L, k) for L in self.layers for k in L.__slots__]
        return sum(t.numel() * t.element_size() for t in ts if t is not None)

    # ---- cache -------------------------------------------------------------------------------------------------------------------
    def cache_bytes_per_token(self) -> int:
        el = torch.empty(0, dtype=self.dtype).element_size()
        return sum(L.mixer.kv_row * el for L in self.hp.layers if isinstance(L.mixer, LatentMixer) and L.mixer.kv_from is None)

    def make_cache(self, n_slots: int, n_seqs: int):
        """Paged rows of ``n_slots`` tokens for the layers that store latents, one state row per sequence slot for the rest."""
        from ..runtime.cache import HybridCache
        d, taps = self.hp.n_embd, self.hp.taps
        rows: List[Any] = []
        for L in self.hp.layers:
            m = L.mixer
            rows.append((m.kv_row if m.kv_from is None else ("layer", m.kv_from)) if isinstance(m, LatentMixer) else None)
        state = {"conv": [((taps - 1, d), self.dtype)] * self.hp.n_layer,
                 "gru": [((L.mixer.width,), torch.float32) if isinstance(L.mixer, GruMixer) else None for L in self.hp.layers]}
        return HybridCache(rows, state, n_slots, n_seqs, self.dtype, self.device, self.block_size)

    # ---- forward -----------------------------------------------------------------------------------------------------------------
    def _attention(self, i: int, L: _Layer, m: LatentMixer, hc: torch.Tensor, b: ForwardBatch, cache) -> torch.Tensor:
        H, dn, dr, r = m.heads, m.dim, m.rot_dim, m.kv_rank
        T = hc.shape[0]
        qkv = ops.linear(hc, L.w_in)
        nq = H * (dn + dr)
        q, ckv = qkv[:, :nq], (qkv[:, nq:] if m.kv_from is None else None)
        rows, rope = cache[i], self.rope[(dr, m.rope_base)]
        if b.max_q_len > 1 and L.w_kv_b is not None and ops.use_native(q) and \
                ops.nat().mha_prefill_ok(T, dn, dr, m.vdim, r, self.block_size, b.attn_meta, m.window):
            ops.mla_qkv_post(q, ckv, L.kv_norm, self.hp.eps, rope, b.positions, b.slot_mapping, rows, None, H, dn, dr, r, True)
            return ops.nat().mha_prefill(q, rows, L.w_kv_b, b.block_tables, b.seq_lens, b.q_start, m.scale, H, self.block_size, b.attn_meta,
                                         m.window)
        q_full = torch.empty(T, H, r + dr, dtype=hc.dtype, device=hc.device)
        q_nope = ops.mla_qkv_post(q, ckv, L.kv_norm, self.hp.eps, rope, b.positions, b.slot_mapping, rows, q_full, H, dn, dr, r, True)
        ops.q_absorb(q_nope, L.w_uk, q_full, r)
        o_lat = ops.mla_attention(q_full, rows, b.block_tables, b.seq_lens, b.q_start, m.scale, r, self.block_size, b.max_q_len, b.attn_meta,
                                  m.window)
        return ops.v_up(o_lat, L.w_uv)

    def _experts(self, L: _Layer, e: Experts, h: torch.Tensor):
        ids, wts = ops.moe_gate(h, L.router, None, e.top, 1, 1, 1.0, True, False, logit_bias=L.router_b)
        y, dest = ops.moe_routed(h, ids, wts, L.w_gate_exps, L.w_up_exps, L.w_down_exps)
        return y, dest, wts

    @torch.no_grad()
    def forward(self, batch: ForwardBatch, cache) -> torch.Tensor:
        """fp32 logits [len(out_rows), n_vocab]; ``cache`` is a ``HybridCache`` of this model."""
        hp, b = self.hp, batch
        T = b.tokens.shape[0]
        single = b.max_q_len == 1 and b.seq_lens.shape[0] == T       # row t is sequence t's only token
        conv_state, gru_state = cache.state["conv"], cache.state["gru"]

        def nxt(i):                   # what follows the residual update: layer i's norm and, for single tokens, its convolution
            if i == hp.n_layer:
                return None
            L = self.layers[i]
            return L.norm, hp.eps, ((L.conv, conv_state[i], b.seq_slots, b.positions) if single else None)

        x, h, hc = ops.embed_norm(self.embed, b.tokens, self.embed_norm, hp.eps, nxt(0))
        for i, (L, s) in enumerate(zip(self.layers, hp.layers)):
            if hc is None:
                hc = ops.causal_conv(h, L.conv, conv_state[i], b.seq_slots, b.positions, b.q_start)
            gates = ops.linear(h, L.w_gates)
            if isinstance(s.mixer, LatentMixer):
                y = self._attention(i, L, s.mixer, hc, b, cache)
            else:
                y = ops.mingru(ops.linear(hc, L.w_in), L.zb, L.xb, gru_state[i], b.seq_slots, b.positions, b.q_start, single)
            o = ops.linear(y, L.w_o)
            moe = self._experts(L, s.mlp, h) if s.mlp is not None else None
            x, h, hc = ops.block_update(x, hp.residual_mult, o, gates, L.b1, L.b2, moe, nxt(i + 1))
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
