"""What one layer's token mixer computes: sizes, constants and small parameter tensors, shared by the kernels and the reference ops."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch


@dataclass
class StateMix:
    """A mixer with a matrix state per head: S <- diag(decay) S; u = s (v - [delta] S^T k); S <- S + k u^T; o = S^T q + skip v.

    ``kind``  "delta": q, k unit vectors, decay exp(neg_a softplus(. + bias)) per key channel, s = sigmoid(.), norm per head, sigmoid gate;
    "linear": decay sigmoid(. + bias)^inv_tau per key channel, s = 1, norm per head, silu gate;
    "ssd": s = softplus(. + bias), decay exp(neg_a s) per head, silu gate, then a norm over ``norm_groups`` parts of the row;
    "hgrn": decay f = lower + (1 - lower) sigmoid(. + bias) per key channel, k = 1 - f, silu on q, s = 1, norm per head, no gate;
    "mlstm": decay and s per head from two log gates i = cap tanh((. + bias) / cap) and f = log sigmoid(cap tanh((. + bias) / cap)) (``bias``: i, f), relative to a running
    maximum top <- max(f + top, i) that starts at 0: decay exp(f + top_old - top), s exp(i - top).  What the k add up to decays and grows like the
    state; o is divided by max(|that sum . q|, exp(-top)) + 1e-6, then a norm per head (``norm_w`` [heads * vdim]), sigmoid gate.
    ``*_off``: columns of the projection.  Columns conv0 .. conv0 + n of it pass a causal convolution of ``taps`` taps (0: none) and silu."""
    kind: str
    heads: int
    dim: int                                    # key channels
    vdim: int
    rep: int = 1                                # heads that share a q / k head
    q_off: int = 0
    k_off: int = 0
    v_off: int = 0
    s_off: int = 0
    taps: int = 0
    conv0: int = 0
    conv_w: Optional[torch.Tensor] = None       # [taps, n] fp32, last tap = current token
    conv_b: Optional[torch.Tensor] = None
    bias: Optional[torch.Tensor] = None
    neg_a: Optional[torch.Tensor] = None        # [heads]
    skip: Optional[torch.Tensor] = None         # [heads]
    norm_w: Optional[torch.Tensor] = None
    norm_groups: int = 1
    q_scale: float = 1.0
    inv_tau: float = 1.0
    eps: float = 1e-6
    out_scale: float = 1.0
    lower: Optional[torch.Tensor] = None        # [heads * dim] fp32, "hgrn"
    gate_cap: float = 0.0                       # "mlstm"


@dataclass
class Gqa:
    """Grouped-query attention with normed q and k (norm weights None: no norm), RoPE on the first ``rot`` dimensions (pairs (i, i + rot / 2), or
    with ``neighbours`` (2 i, 2 i + 1)), with ``unit`` q and k over their root mean square after it, scores * scale, softcap (0: none), a
    causal mask with a sliding window and / or chunks (0: none), and with ``sink`` one more key without a value, of score 0 or
    ``sink_w[head]``.

    ``pool`` > 0: beside its window a query sees one key and value for every block of ``pool`` positions that lies wholly before the window,
    the means of the block's cached rows.  ``v_mix`` is not None: the cached values are (1 - v_mix) v + v_mix v_first.  ``gate_each``: the
    gate holds a column per head and value channel instead of one per head."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    rot: int
    scale: float
    q_norm: Optional[torch.Tensor] = None
    k_norm: Optional[torch.Tensor] = None
    softcap: float = 0.0
    window: int = 0
    chunk: int = 0
    sink: bool = False
    eps: float = 1e-6
    out_scale: float = 1.0
    sink_w: Optional[torch.Tensor] = None       # [heads] fp32
    neighbours: bool = False
    unit: bool = False
    pool: int = 0
    v_mix: Optional[float] = None
    gate_each: bool = False

    @property
    def kv_row(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)

    def pool_rows(self, block_size: int) -> int:
        """Pooled rows kept per cache block: those of the pooled blocks that end in it (padded so that cache blocks stay 16-byte multiples)."""
        if not self.pool:
            return 0
        n = (block_size + self.pool - 1) // self.pool
        return n if n * self.kv_row % 8 == 0 else (n + 7) // 8 * 8


@dataclass
class SelectiveScan:
    """A state-space recurrence with a decay per channel and state: S[c, n] <- exp(dt_c neg_a[c, n]) S[c, n] + dt_c x_c B_n,
    y_c = (sum_n S[c, n] C_n + skip_c x_c) silu(z_c) out_scale, dt = softplus(. + dt_bias).  ``channels`` and ``state`` are multiples of 8 (a model
    pads with zero weights)."""
    channels: int
    state: int
    neg_a: torch.Tensor                         # [channels, state] fp32
    skip: torch.Tensor                          # [channels] fp32
    dt_bias: torch.Tensor                       # [channels] fp32
    out_scale: float = 1.0


@dataclass
class RowNorms:
    """What an updated residual row turns into: row / rms * w1, and with ``w2`` row / rms * w2 as well; ``w1`` None: the row itself in the
    activation type.  ``groups``: equal parts of the row, each over its own rms."""
    eps: float = 0.0
    w1: Optional[torch.Tensor] = None
    w2: Optional[torch.Tensor] = None
    groups: int = 1
