"""What the models of folder checkpoints share: tensor intake, rotations, stacked projections."""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Callable, Dict, Iterator, List, Optional, Sequence, Tuple

import torch

ALIGN = 8                          # columns: 16 bytes of bf16


@dataclass(frozen=True)
class Yarn:
    factor: float
    original: float
    fast: float
    slow: float


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    yarn: Optional[Yarn] = None
    stretch: float = 1.0             # every frequency is divided by it


def fits(shape: Sequence[int], want: Sequence[Optional[int]]) -> bool:
    return len(shape) == len(want) and all(w is None or s == w for s, w in zip(shape, want))


def checked_tensors(directory: str, table: Dict[str, Tuple[Optional[int], ...]], unused: Callable[[str], bool] = lambda n: False
                    ) -> Iterator[Tuple[str, torch.Tensor]]:
    """(name, CPU tensor) of every tensor of ``table`` (name -> shape, None: any size) from the folder's safetensors file(s); no other
    tensors may be there but those ``unused`` allows."""
    from ..gguf.convert_hf import Checkpoint
    ck = Checkpoint(directory)
    try:
        have = set(ck.names())
        missing = [n for n in table if n not in have]
        if missing:
            raise KeyError(f"checkpoint is missing {len(missing)} tensors, e.g. {missing[:3]}")
        extra = sorted(n for n in have - set(table) if not unused(n))
        if extra:
            raise ValueError(f"checkpoint has {len(extra)} tensors the model does not use, e.g. {extra[:3]}")
        for name, shape in table.items():
            t = ck.get(name)
            if not fits(t.shape, shape):
                raise ValueError(f"{name}: shape {tuple(t.shape)} != expected {shape}")
            yield name, t
    finally:
        ck.close()


def rope_table(n_pos: int, rot: Rotation, device) -> torch.Tensor:
    """[n_pos, dims / 2, 2] fp32 (cos, sin), with linear stretching or YaRN's blend of stretched and plain frequencies and its magnitude factor."""
    i = torch.arange(rot.dims // 2, dtype=torch.float64)
    f, mult = rot.base ** (-2.0 * i / rot.dims) / rot.stretch, 1.0
    if rot.yarn is not None:
        y = rot.yarn
        at = lambda turns: rot.dims * math.log(y.original / (2 * math.pi * turns)) / (2 * math.log(rot.base))       # noqa: E731
        lo, hi = max(math.floor(at(y.fast)), 0), min(math.ceil(at(y.slow)), rot.dims - 1)
        ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
        f, mult = f / y.factor * ramp + f * (1 - ramp), 0.1 * math.log(y.factor) + 1
    a = torch.arange(n_pos, dtype=torch.float64)[:, None] * f
    return torch.stack([torch.cos(a) * mult, torch.sin(a) * mult], -1).float().contiguous().to(device)


def up(n: int) -> int:
    return (n + ALIGN - 1) // ALIGN * ALIGN


def stack_rows(parts: Sequence[Tuple[str, torch.Tensor]]) -> Tuple[torch.Tensor, Dict[str, int]]:
    """Matrices of equal width over one another, each starting at a multiple of 8 rows (zero rows between); (matrix, first row of each)."""
    off, n = {}, 0
    for k, w in parts:
        off[k] = n
        n += up(w.shape[0])
    out = torch.zeros(n, parts[0][1].shape[1], dtype=parts[0][1].dtype, device=parts[0][1].device)
    for k, w in parts:
        out[off[k]:off[k] + w.shape[0]] = w
    return out, off


def block_diagonal(parts: Sequence[torch.Tensor]) -> Tuple[torch.Tensor, List[int]]:
    """Matrices along the diagonal of one, rows and columns of each starting at multiples of 8; (matrix, first row of each)."""
    rows, cols = [0], [0]
    for w in parts:
        rows.append(rows[-1] + up(w.shape[0]))
        cols.append(cols[-1] + up(w.shape[1]))
    out = torch.zeros(rows[-1], cols[-1], dtype=parts[0].dtype, device=parts[0].device)
    for w, r, c in zip(parts, rows, cols):
        out[r:r + w.shape[0], c:c + w.shape[1]] = w
    return out, rows[:-1]
