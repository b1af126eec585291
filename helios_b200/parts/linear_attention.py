"""A recurrent mixer: linear attention with a fixed decay per head and no softmax.

q, k (heads x dk) and v (heads x dv) are projections of the mixer's input; optionally all
three pass silu (``activation``), optionally q and k are rotated by a position encoding on
their first ``rotary_dim`` values (value i paired with value i + rotary_dim / 2); k is
multiplied by ``key_scale``.  Per token and head, with the head's constant a:

    S <- a S + k v^T          (S is [dk, dv])
    o  = S^T q

o is RMS-normed, per head without a weight (``norm`` "head") or over the whole row of heads
with a weight per channel ("row"), multiplied by a gate of the input (``gate`` "silu" or
"sigmoid" of W_g h), and projected out.  A request's slot holds S (float32); nothing is kept
per token.  Everything between the projections and the gated output is float32.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..csrc import ops
from .base import StateSpec, WeightSpec, register_part
from .side_by_side import BranchMixer


class FixedDecayMixer(BranchMixer):
    def __init__(self, width: int, heads: int, dk: int, dv: int, decay, eps: float, *, key_scale: float = 1.0,
                 activation: str = "none", position=None, rotary_dim: int = 0, norm: str = "head",
                 gate: str = "silu", names=("q", "k", "v", "g", "o", "norm")) -> None:
        """``decay``: a number per head in [0, 1].  ``names``: the tensors below the part's
        prefix (projections q, k, v, gate, output, and the norm's weight with ``norm`` "row")."""
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        if activation not in ops.LINEAR_ATTENTION_ACTIVATIONS or norm not in ops.LINEAR_ATTENTION_NORMS \
                or gate not in ops.LINEAR_ATTENTION_GATES:
            raise ValueError(f"activation {activation!r} / norm {norm!r} / gate {gate!r}")
        if (position is None) != (not rotary_dim) or rotary_dim % 2 or rotary_dim > dk:
            raise ValueError(f"a rotation needs an encoding and an even rotary_dim of at most {dk}")
        if dk > 256 or dv > 256:
            raise ValueError(f"heads of {dk} x {dv} are not supported (at most 256)")
        self.width, self.heads, self.dk, self.dv = width, heads, dk, dv
        self.decay_values = [float(d) for d in decay]
        self.eps, self.key_scale = float(eps), float(key_scale)
        self.activation, self.position, self.rotary_dim = activation, position, int(rotary_dim)
        self.norm, self.gate = norm, gate
        self.names = tuple(names)
        self.in_columns = heads * (2 * dk + 2 * dv)
        self.out_columns = heads * dv
        self.decay_powers = self.norm_weight = None

    def state_spec(self) -> StateSpec:
        return StateSpec((self.heads * self.dk * self.dv,), torch.float32)

    def kernel_libraries(self, dtype):
        return ops.linear_libraries(dtype, self.width) + ("linear_attention",)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        nq, nk, nv, ng, no, nn = self.names
        qk, v = self.heads * self.dk, self.heads * self.dv
        specs = {nq: WeightSpec((qk, self.width)), nk: WeightSpec((qk, self.width)),
                 nv: WeightSpec((v, self.width)), ng: WeightSpec((v, self.width)),
                 no: WeightSpec((self.width, v))}
        if self.norm == "row":
            specs[nn] = WeightSpec((v,), kind="vector", init="ones_jitter")
        return specs

    def in_matrices(self, tensors: Dict[str, torch.Tensor]) -> List[torch.Tensor]:
        return [tensors[n] for n in self.names[:4]]

    def out_matrix(self, tensors: Dict[str, torch.Tensor]) -> torch.Tensor:
        return tensors[self.names[4]]

    def bind_rest(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.decay_powers = ops.decay_power_table(self.decay_values, tensors[self.names[4]].device)
        if self.norm == "row":
            self.norm_weight = tensors[self.names[5]].contiguous()

    def run(self, ctx, rows, col0, out, factor, cache, state) -> None:
        qk, v = self.heads * self.dk, self.heads * self.dv
        cos, sin = self.position.tables(ctx) if self.position is not None else (None, None)
        ops.linear_attention(ctx, rows, (col0, col0 + qk, col0 + 2 * qk, col0 + 2 * qk + v), state,
                             self.decay_powers, self.heads, self.dk, self.dv, out, cos=cos, sin=sin,
                             key_scale=self.key_scale, activation=self.activation, norm=self.norm,
                             norm_weight=self.norm_weight, gate=self.gate, eps=self.eps, factor=factor)


register_part("mixer", "fixed_decay", FixedDecayMixer)
