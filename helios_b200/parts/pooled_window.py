"""Grouped-query window attention that sees older tokens as means of whole blocks.

q, k and v are projections of the mixer's input, each followed by a short causal convolution
over time per channel (``taps``; 0: none); q and k are RMS-normed per head with a weight
shared by the heads, then rotated on their first ``rotary_dim`` values (value i paired with
value i + rotary_dim / 2).  Position i sees

    the tokens j with 0 <= i - j < window, and
    every block of ``pool`` tokens [b pool, (b + 1) pool) that ends at or before i - window,
    as ONE key and ONE value: the means of the block's keys and values as the cache holds them

under one softmax of q . k * scale (``pool`` 0: the window alone).  Tokens stay in the pages
for as long as the window or their own unfinished block needs them; a block's key and value
are written once, in the step that brings its last token, to pages of their own.
"""
from __future__ import annotations

from typing import Dict, List, Optional

import torch

from ..csrc import ops
from .base import PagedCacheSpec, StateSpec, WeightSpec, register_part
from .side_by_side import BranchMixer


class PooledWindowAttention(BranchMixer):
    def __init__(self, width: int, num_heads: int, num_kv_heads: int, head_dim: int, value_dim: int,
                 scale: float, window: int, pool: int, eps: float, position, rotary_dim: int, taps: int = 0,
                 names=("q", "k", "v", "o", "q.norm", "k.norm"), conv_suffix: str = ".conv") -> None:
        if num_heads % num_kv_heads:
            raise ValueError(f"{num_heads} query heads are not a multiple of {num_kv_heads} KV heads")
        if not 0 < head_dim <= 256 or not 0 < value_dim <= 256:
            raise ValueError(f"heads of {head_dim} / {value_dim} values are not supported (at most 256)")
        if rotary_dim % 2 or rotary_dim > head_dim:
            raise ValueError(f"rotary_dim {rotary_dim} must be even and at most {head_dim}")
        if window < 1 or pool < 0 or taps < 0:
            raise ValueError(f"window {window} / pool {pool} / taps {taps}")
        self.width, self.num_heads, self.num_kv_heads = width, num_heads, num_kv_heads
        self.head_dim, self.value_dim = head_dim, value_dim
        self.scale, self.eps = float(scale), float(eps)
        self.window, self.pool, self.taps = int(window), int(pool), int(taps)
        self.position, self.rotary_dim = position, int(rotary_dim)
        self.names, self.conv_suffix = tuple(names), conv_suffix
        self.in_columns = num_heads * head_dim + num_kv_heads * (head_dim + value_dim)
        self.out_columns = num_heads * value_dim
        self.q_weight = self.k_weight = self.conv_weight = None

    def cache_spec(self) -> PagedCacheSpec:
        vd = None if self.value_dim == self.head_dim else self.value_dim
        # an unfinished block's tokens are still wanted when the window has passed them
        return PagedCacheSpec(self.num_kv_heads, self.head_dim, max(self.window, self.pool), value_dim=vd,
                              pool=self.pool)

    def state_spec(self) -> Optional[StateSpec]:
        """The last taps - 1 inputs of the convolutions, oldest first per channel."""
        n = self.in_columns * max(0, self.taps - 1)
        return StateSpec((n,), torch.float32) if n else None

    def kernel_libraries(self, dtype):
        return ops.linear_libraries(dtype, self.width) + ops.pooled_attention_libraries(
            dtype, self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim)

    def weight_specs(self) -> Dict[str, WeightSpec]:
        nq, nk, nv, no, nqn, nkn = self.names
        q, k = self.num_heads * self.head_dim, self.num_kv_heads * self.head_dim
        v = self.num_kv_heads * self.value_dim
        specs = {nq: WeightSpec((q, self.width)), nk: WeightSpec((k, self.width)), nv: WeightSpec((v, self.width)),
                 nqn: WeightSpec((self.head_dim,), kind="vector", init="ones_jitter"),
                 nkn: WeightSpec((self.head_dim,), kind="vector", init="ones_jitter"),
                 no: WeightSpec((self.width, self.num_heads * self.value_dim))}
        if self.taps:
            for n in (nq, nk, nv):
                specs[n + self.conv_suffix] = WeightSpec((specs[n].shape[0], self.taps), kind="vector", std=0.3)
        return specs

    def in_matrices(self, tensors: Dict[str, torch.Tensor]) -> List[torch.Tensor]:
        return [tensors[n] for n in self.names[:3]]

    def out_matrix(self, tensors: Dict[str, torch.Tensor]) -> torch.Tensor:
        return tensors[self.names[3]]

    def bind_rest(self, tensors: Dict[str, torch.Tensor]) -> None:
        self.q_weight, self.k_weight = tensors[self.names[4]].contiguous(), tensors[self.names[5]].contiguous()
        if self.taps:
            self.conv_weight = torch.cat([tensors[n + self.conv_suffix] for n in self.names[:3]]).contiguous()

    def run(self, ctx, rows, col0, out, factor, cache, state) -> None:
        cos, sin = self.position.tables(ctx)
        pooled = cache.pooled
        q = ops.conv_norm_rotate_write(ctx, rows, col0, self.conv_weight, state, self.q_weight, self.k_weight,
                                       self.eps, cos, sin, cache, self.num_heads, self.num_kv_heads,
                                       self.head_dim, self.value_dim)
        if pooled is not None and cache.write:
            ops.pool_blocks(ctx, cache, self.pool)
        ops.pooled_attention(ctx, q, cache, self.num_heads, self.num_kv_heads, self.head_dim, self.value_dim,
                             self.window, self.pool, self.scale, out, factor)


register_part("mixer", "pooled_window", PooledWindowAttention)
