"""Device memory behind the block tables and sequence slots, for models whose layers do not all store the same rows.

``SplitCache``   one latent tensor per device of a layer-split model.
``HybridCache``  per-layer row widths, layers that read another layer's rows, and a state row per sequence slot for what is not
                 paged (recurrent states, convolution inputs).

Both are indexed by layer and copy blocks for the allocator's copy-on-write and defragmentation moves.
"""
from __future__ import annotations

from typing import Any, Dict, List, Optional, Sequence, Tuple

import numpy as np
import torch

from .. import ops


class SplitCache:
    """Latent cache of a layer-split model: one [layers-on-device, n_slots, row] tensor per device; ``cache[il]`` is the
    layer's slice on its own device."""

    def __init__(self, layer_dev, n_slots: int, row: int, dtype, block_size: int):
        self.block_size = block_size
        self.by_dev: Dict[torch.device, torch.Tensor] = {}
        self.index: List[Tuple[torch.device, int]] = []
        counts: Dict[torch.device, int] = {}
        for d in layer_dev:
            self.index.append((d, counts.get(d, 0)))
            counts[d] = counts.get(d, 0) + 1
        for d, n in counts.items():
            self.by_dev[d] = torch.zeros(n, n_slots, row, dtype=dtype, device=d)

    def __len__(self) -> int:
        return len(self.index)

    def __getitem__(self, il: int) -> torch.Tensor:
        d, i = self.index[il]
        return self.by_dev[d][i]

    def copy_blocks(self, src: np.ndarray, dst: np.ndarray) -> None:
        for d, t in self.by_dev.items():
            s = torch.from_numpy(np.ascontiguousarray(src)).to(d)
            e = torch.from_numpy(np.ascontiguousarray(dst)).to(d)
            if d.type == "cuda":
                with torch.cuda.device(d):
                    ops.kv_block_copy(t, s, e, self.block_size)
            else:
                ops.kv_block_copy(t, s, e, self.block_size)


class HybridCache:
    """One entry per layer, or per layer run where a model runs a layer several times.  ``rows[i]``: width of layer i's paged rows, ``("layer", j)`` for a layer that reads layer j's, None for none.
    ``state[name][i]``: (shape, dtype) of what one sequence keeps for layer i under that name, or None.

    ``cache[i]`` is the [n_slots, width] tensor layer i reads; ``cache.state[name][i]`` the [n_seqs, *shape] tensor.  State rows are
    never cleared: kernels start a sequence's first token from zeros.  ``pooled[i]`` > 0: layer i also keeps that many rows of the same
    width per block, ``cache.pool[i]`` [blocks * rows, width], which go where the block goes."""

    def __init__(self, rows: Sequence[Any], state: Dict[str, Sequence[Optional[Tuple[Tuple[int, ...], torch.dtype]]]], n_slots: int,
                 n_seqs: int, dtype: torch.dtype, device: torch.device, block_size: int, pooled: Optional[Sequence[int]] = None):
        self.block_size = block_size
        self.own: List[torch.Tensor] = []
        self._rows: List[Optional[torch.Tensor]] = []
        self.pool_rows = list(pooled) if pooled is not None else [0] * len(rows)
        self.pool = [torch.zeros(n_slots // block_size * n, r, dtype=dtype, device=device) if n else None for n, r in zip(self.pool_rows, rows)]
        for r in rows:
            if r is None:
                self._rows.append(None)
            elif isinstance(r, tuple):
                self._rows.append(self._rows[r[1]])
            else:
                t = torch.zeros(n_slots, r, dtype=dtype, device=device)
                self.own.append(t)
                self._rows.append(t)
        self.state = {k: [None if s is None else torch.zeros((n_seqs,) + tuple(s[0]), dtype=s[1], device=device) for s in v]
                      for k, v in state.items()}

    def __len__(self) -> int:
        return len(self._rows)

    def __getitem__(self, il: int) -> Optional[torch.Tensor]:
        return self._rows[il]

    def copy_blocks(self, src: np.ndarray, dst: np.ndarray) -> None:
        if not self.own:
            return
        dev = self.own[0].device
        s = torch.from_numpy(np.ascontiguousarray(src)).to(dev)
        d = torch.from_numpy(np.ascontiguousarray(dst)).to(dev)
        for t in self.own:
            ops.kv_block_copy(t[None], s, d, self.block_size)
        for t, n in zip(self.pool, self.pool_rows):
            if t is not None:
                ops.kv_block_copy(t[None], s, d, n)
