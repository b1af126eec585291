"""A recurrent mixer: linear attention whose decay is a vector that depends on the token.

q, k (heads x dk) and v (heads x dv) are projections of the mixer's input h; q is multiplied by
``q_scale``.  Per token and head, with a decay for every key channel that comes from a low-rank
projection,

    a  = sigmoid(W_a2 (W_a1 h) + b)^(1 / tau)        (heads x dk)
    S <- diag(a) S + k v^T                           (S is [dk, dv])
    o  = S^T q

Each head's o is RMS-normed over its dv values with one weight for all heads, multiplied by
silu(W_g h), and projected out.  A request's slot holds S (float32); nothing is kept per token.
Everything between the projections and the gated output is float32: the decays themselves (the
product with W_a2 included), the recurrence, the norm, the gate.
"""
from __future__ import annotations

from typing import Dict, List

import torch

from ..csrc import ops
from .base import StateSpec, WeightSpec, register_part
from .side_by_side import BranchMixer


class ChannelDecayMixer(BranchMixer):
    def __init__(self, width: int, heads: int, dk: int, dv: int, decay_rank: int, tau: float, eps: float, *,
                 q_scale: float = 1.0, names=("q", "k", "v", "g", "a1", "a2", "o", "norm"),
                 bias_suffix: str = ".b") -> None:
        """``decay_rank``: rows of W_a1.  ``names``: the tensors below the part's prefix
        (projections q, k, v, gate; the decay's two matrices, the second with a bias; output
        projection; the norm's weight)."""
        if dk > 256 or dv > 256 or decay_rank > 256:
            raise ValueError(f"heads of {dk} x {dv} with a decay of rank {decay_rank} are not supported (at most 256)")
        if not tau > 0:
            raise ValueError(f"tau {tau} must be positive")
        self.width, self.heads, self.dk, self.dv = width, heads, dk, dv
        self.decay_rank, self.tau = int(decay_rank), float(tau)
        self.eps, self.q_scale = float(eps), float(q_scale)
        self.names, self.bias_suffix = tuple(names), bias_suffix
        self.in_columns = heads * (2 * dk + 2 * dv) + self.decay_rank
        self.out_columns = heads * dv
        self.w_a2 = self.b_a2 = self.norm_weight = None

    def state_spec(self) -> StateSpec:
        return StateSpec((self.heads * self.dk * self.dv,), torch.float32)

    def kernel_libraries(self, dtype):
        return ops.linear_libraries(dtype, self.width) + ("gated_linear_attention",) \
            + (("linear_attention",) if self.dv > 128 else ())

    def weight_specs(self) -> Dict[str, WeightSpec]:
        nq, nk, nv, ng, na1, na2, no, nn = self.names
        qk, v = self.heads * self.dk, self.heads * self.dv
        return {nq: WeightSpec((qk, self.width)), nk: WeightSpec((qk, self.width)),
                nv: WeightSpec((v, self.width)), ng: WeightSpec((v, self.width)),
                na1: WeightSpec((self.decay_rank, self.width)), na2: WeightSpec((qk, self.decay_rank)),
                na2 + self.bias_suffix: WeightSpec((qk,), kind="vector", init="normal", std=1.0),
                no: WeightSpec((self.width, v)),
                nn: WeightSpec((self.dv,), kind="vector", init="ones_jitter")}

    def in_matrices(self, tensors: Dict[str, torch.Tensor]) -> List[torch.Tensor]:
        return [tensors[n] for n in self.names[:5]]

    def out_matrix(self, tensors: Dict[str, torch.Tensor]) -> torch.Tensor:
        return tensors[self.names[6]]

    def bind_rest(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.w_a2 = tensors[self.names[5]].contiguous()
        self.b_a2 = tensors[self.names[5] + self.bias_suffix].contiguous()
        self.norm_weight = tensors[self.names[7]].contiguous()

    def run(self, ctx, rows, col0, out, factor, cache, state) -> None:
        qk, v = self.heads * self.dk, self.heads * self.dv
        offsets = (col0, col0 + qk, col0 + 2 * qk, col0 + 2 * qk + v, col0 + 2 * qk + 2 * v)
        ops.gated_linear_attention(ctx, rows, offsets, self.w_a2, self.b_a2, self.tau, state, self.heads, self.dk,
                                   self.dv, self.norm_weight, self.eps, out, q_scale=self.q_scale, factor=factor)


register_part("mixer", "channel_decay", ChannelDecayMixer)
