"""Two mixers that read the same input side by side, each with a factor on its output:

    left_scale * left(h) + right_scale * right(h)

The matrices at either end are shared: ONE projection makes the rows both read, and ONE
product takes both outputs, which the mixers leave beside each other in one row, each times
its factor (applied in float32 where the mixer writes its output, so a row is rounded once).
A mixer that can run so is a ``BranchMixer``; it also runs alone.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..csrc import ops
from .base import Mixer, StateSpec, WeightSpec, register_part


def _up8(n: int) -> int:
    return -(-n // 8) * 8


class BranchMixer(Mixer):
    """A mixer of the form W_o f(W_in h).  ``in_columns``: what its share of a fused projection
    is wide; ``out_columns``: what ``W_o`` takes.  Its state, if any, is one float32 vector a
    request."""

    width: int
    in_columns: int
    out_columns: int
    w_in: Optional[torch.Tensor] = None
    w_o: Optional[torch.Tensor] = None

    def in_matrices(self, tensors: Dict[str, torch.Tensor]) -> List[torch.Tensor]:
        """The matrices of its share of the projection, in the order of its columns."""
        raise NotImplementedError

    def out_matrix(self, tensors: Dict[str, torch.Tensor]) -> torch.Tensor:
        raise NotImplementedError

    def bind_rest(self, tensors: Dict[str, torch.Tensor]) -> None:
        """Everything but the matrices above."""

    def run(self, ctx, rows: torch.Tensor, col0: int, out: torch.Tensor, factor: float, cache, state) -> None:
        """``rows`` [T, .] the projection, this mixer's share from column ``col0`` on; writes
        ``factor`` times what W_o takes into ``out`` [T, >= out_columns] (rows may be strided)."""
        raise NotImplementedError

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_in, self.w_o = _fused_matrices([self], [tensors], self.width)
        self.bind_rest(tensors)

    def forward(self, ctx, x: torch.Tensor, cache, state=None) -> torch.Tensor:
        rows = ops.linear(x, self.w_in)
        out = _rows_for([self.out_columns], self.w_o.shape[1], rows)
        self.run(ctx, rows, 0, out, 1.0, cache, state)
        return ops.linear(out, self.w_o)


def _fused_matrices(mixers, tensors, width: int):
    """(W_in, W_o) of one or more branches: input matrices stacked, every branch's columns
    beginning at a multiple of 8 (16-byte pieces; the gaps are zero rows and columns)."""
    rows, cols = [], []
    for mx, t in zip(mixers, tensors):
        mats = mx.in_matrices(t)
        gap = _up8(mx.in_columns) - mx.in_columns
        if gap:
            mats = mats + [mats[0].new_zeros((gap, width))]
        rows += mats
        out = mx.out_matrix(t)
        gap = _up8(mx.out_columns) - mx.out_columns
        cols.append(torch.cat([out, out.new_zeros((width, gap))], dim=1) if gap else out)
    return torch.cat(rows, dim=0).contiguous(), torch.cat(cols, dim=1).contiguous()


def _rows_for(out_columns: List[int], total: int, like: torch.Tensor) -> torch.Tensor:
    make = torch.zeros if any(n % 8 for n in out_columns) else torch.empty
    return make((like.shape[0], total), dtype=like.dtype, device=like.device)


class SideBySideMixer(Mixer):
    def __init__(self, left: BranchMixer, right: BranchMixer, left_scale: float, right_scale: float,
                 names=("left.", "right.")) -> None:
        if left.width != right.width:
            raise ValueError(f"mixers of widths {left.width} and {right.width} cannot read the same input")
        if left.cache_spec() is not None and right.cache_spec() is not None:
            raise ValueError("only one of two mixers side by side may keep pages")
        self.branches = (left, right)
        self.scales = (float(left_scale), float(right_scale))
        self.names = tuple(names)
        self.width = left.width
        self.w_in = self.w_o = None
        self._state_floats = [0 if (s := b.state_spec()) is None else int(s.shape[0]) for b in self.branches]

    def cache_spec(self):
        return self.branches[0].cache_spec() or self.branches[1].cache_spec()

    def state_spec(self) -> Optional[StateSpec]:
        n = sum(self._state_floats)
        return StateSpec((n,), torch.float32) if n else None

    def kernel_libraries(self, dtype):
        return tuple(n for b in self.branches for n in b.kernel_libraries(dtype))

    def weight_specs(self) -> Dict[str, WeightSpec]:
        return {prefix + name: spec for prefix, b in zip(self.names, self.branches)
                for name, spec in b.weight_specs().items()}

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        own = [{n[len(p):]: t for n, t in tensors.items() if n.startswith(p)} for p in self.names]
        self.w_in, self.w_o = _fused_matrices(self.branches, own, self.width)
        for b, t in zip(self.branches, own):
            b.bind_rest(t)

    def forward(self, ctx, x: torch.Tensor, cache, state=None) -> torch.Tensor:
        rows = ops.linear(x, self.w_in)
        out = _rows_for([b.out_columns for b in self.branches], self.w_o.shape[1], rows)
        col = at = floats = 0
        for b, scale, n in zip(self.branches, self.scales, self._state_floats):
            b.run(ctx, rows, col, out[:, at:at + b.out_columns], scale,
                  cache if b.cache_spec() is not None else None, state[:, floats:floats + n] if n else None)
            col, at, floats = col + _up8(b.in_columns), at + _up8(b.out_columns), floats + n
        return ops.linear(out, self.w_o)


register_part("mixer", "side_by_side", SideBySideMixer)
