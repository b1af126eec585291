"""Attention over a low-rank latent cache.

Per token the mixer keeps ONE row: the latent c (``rank`` values, RMS-normed) and a rotated
key part r (``rot`` values) that all heads share.  Head h's key is [W_uk[h] c | r] and its
value W_uv[h] c; a query is [q_nope (``nope`` values) | q_rot (``rot`` values, rotated)] and

    score = (q_nope . W_uk[h] c + q_rot . r) * scale,     softmax over the positions <= own

(or the last ``window`` of them, with a sink or without).

The up-projections are folded into the query and the output, so that the cache is never
expanded: q_lat = W_uk[h]^T q_nope attends the latents themselves, and the head's output is
W_uv[h] (sum_j p_j c_j).  Only a long portion, for which the products over the latents are more work
than making the keys and values per head of the rows it sees, does expand those rows for the step
(``ops.latent_expand_pages``).  Rotary pairs dimension 2i with 2i + 1 over the first
``position.rotary_dim`` of the ``rot`` values.
"""
from __future__ import annotations

from typing import Dict, Optional

import torch

from ..csrc import ops
from .base import LayerCache, Mixer, PagedCacheSpec, WeightSpec, register_part


class LatentAttention(Mixer):
    """Options, each off by default:

    ``q_rank``      the queries go through a latent of their own: c_q = RMSnorm(W_dq h) (weight
                    ``dq.norm``, the mixer's eps), q = W_uq c_q; there is no direct query matrix
    ``pairing``     "neighbours": value 2i of a rotated part is paired with value 2i + 1;
                    "halves": value i with value i + rotary_dim / 2
    ``gate``        "wide" (or True): the concatenated heads are multiplied by sigmoid(W_g h), value
                    by value, before the output projection; "head": W_g has a row per HEAD, and
                    head h's output is multiplied by sigmoid(W_g h)_h
    ``window``      a token sees itself and the ``window`` - 1 tokens before it
    ``sink``        the softmax has one more key, without a value, whose score is a learned number a
                    head (tensor ``sink``), not scaled
    ``own_rows``    False: the mixer has no W_dkv and keeps nothing; it attends the rows that
                    ANOTHER layer keeps (the plan names that layer's cache for this one's run),
                    with up-projections, queries and everything else of its own
    """

    def __init__(self, width: int, heads: int, nope: int, rot: int, vdim: int, rank: int,
                 scale: float, eps: float, position,
                 names=("q", "dkv", "dkv.norm", "uk", "uv", "o"), q_rank: Optional[int] = None,
                 pairing: str = "neighbours", gate=False, own_rows: bool = True,
                 query_names=("dq", "dq.norm", "uq"), gate_name: str = "g", window: Optional[int] = None,
                 sink: bool = False, sink_name: str = "sink") -> None:
        """``position``: the rotary encoding whose tables rotate the ``rot`` parts
        (``position.rotary_dim`` <= rot, even).  ``scale`` multiplies the scores as given.
        ``eps``: of the latents' RMS norms."""
        if position.rotary_dim > rot:
            raise ValueError(f"{position.rotary_dim} rotated dimensions exceed the rotated part of {rot}")
        if pairing not in ops.ROTARY_PAIRINGS:
            raise ValueError(f"pairing {pairing!r} is not one of {sorted(ops.ROTARY_PAIRINGS)}")
        if gate not in (False, True, "wide", "head"):
            raise ValueError(f"gate {gate!r}")
        self.width, self.heads, self.nope, self.rot = width, heads, nope, rot
        self.vdim, self.rank = vdim, rank
        self.scale, self.eps = float(scale), float(eps)
        self.position = position
        self.names = tuple(names)
        self.q_rank = int(q_rank) if q_rank else None
        self.pairing, self.own_rows = pairing, bool(own_rows)
        self.gate = "wide" if gate is True else gate
        self._gate_rows = heads * (vdim if self.gate == "wide" else 1) if self.gate else 0
        self.window, self.sink, self.sink_name = window, bool(sink), sink_name
        self.sink_values = None
        self.query_names, self.gate_name = tuple(query_names), gate_name
        self.w_in = self.w_uq = self.w_uk_t = self.w_uv = self.w_o = self.w_expand = None
        self.norm_weight = self.query_norm_weight = None
        # columns of the fused first projection: [queries or their latent | latent rows | gate]
        self._n_first = self.q_rank or heads * (nope + rot)
        self._lat_col = self._n_first
        self._gate_col = self._lat_col + (rank + rot if self.own_rows else 0)

    def cache_spec(self) -> PagedCacheSpec:
        return PagedCacheSpec(1, self.rank + self.rot, self.window, planes=1)

    def kernel_libraries(self, dtype):
        expand = ops.latent_expand_supported(dtype, self.heads, self.nope + self.rot, self.vdim, self.rank, self.rot, 16)
        return ops.linear_libraries(dtype, self.width) + ("latent_attention",) \
            + (("elementwise",) if self.gate else ()) + (("attention_tc_pooled",) if expand else ())

    def weight_specs(self) -> Dict[str, WeightSpec]:
        q, dkv, norm, uk, uv, o = self.names
        H = self.heads
        specs = {
            uk: WeightSpec((H * self.nope, self.rank)),
            uv: WeightSpec((H * self.vdim, self.rank)),
            o: WeightSpec((self.width, H * self.vdim)),
        }
        if self.q_rank:
            dq, dq_norm, uq = self.query_names
            specs[dq] = WeightSpec((self.q_rank, self.width))
            specs[dq_norm] = WeightSpec((self.q_rank,), kind="vector", init="ones_jitter")
            specs[uq] = WeightSpec((H * (self.nope + self.rot), self.q_rank))
        else:
            specs[q] = WeightSpec((H * (self.nope + self.rot), self.width))
        if self.own_rows:
            specs[dkv] = WeightSpec((self.rank + self.rot, self.width))
            specs[norm] = WeightSpec((self.rank,), kind="vector", init="ones_jitter")
        if self.gate:
            specs[self.gate_name] = WeightSpec((self._gate_rows, self.width))
        if self.sink:
            specs[self.sink_name] = WeightSpec((H,), kind="vector", init="normal", std=0.5)
        return specs

    def bind(self, tensors: Dict[str, torch.Tensor]) -> None:
        q, dkv, norm, uk, uv, o = self.names
        H = self.heads
        mats = [tensors[self.query_names[0]] if self.q_rank else tensors[q]]
        if self.own_rows:
            mats.append(tensors[dkv])
            self.norm_weight = tensors[norm].contiguous()
        if self.gate:
            mats.append(tensors[self.gate_name])
        if len(mats) > 1:
            pad = -sum(m.shape[0] for m in mats) % 8     # output rows stay 16-byte aligned
            if pad:
                mats.append(torch.zeros((pad, self.width), dtype=mats[0].dtype, device=mats[0].device))
        self.w_in = torch.cat(mats, dim=0).contiguous()
        if self.q_rank:
            self.query_norm_weight = tensors[self.query_names[1]].contiguous()
            self.w_uq = tensors[self.query_names[2]].contiguous()
        # [heads, rank, nope]: the matrix that takes a head's q_nope to the latent space
        self.w_uk_t = tensors[uk].view(H, self.nope, self.rank).transpose(1, 2).contiguous()
        self.w_uv = tensors[uv].view(H, self.vdim, self.rank).contiguous()
        self.w_o = tensors[o].contiguous()
        self.w_expand = None
        if ops.latent_expand_supported(self.w_o.dtype, H, self.nope + self.rot, self.vdim, self.rank, self.rot, 16):
            # a row [c | r] -> every head's key [W_uk c | r], then every head's value W_uv c
            key = torch.zeros((H, self.nope + self.rot, self.rank + self.rot), dtype=self.w_o.dtype, device=self.w_o.device)
            key[:, :self.nope, :self.rank] = tensors[uk].view(H, self.nope, self.rank)
            key[:, self.nope:, self.rank:] = torch.eye(self.rot, dtype=key.dtype, device=key.device)
            value = torch.zeros((H * self.vdim, self.rank + self.rot), dtype=key.dtype, device=key.device)
            value[:, :self.rank] = tensors[uv]
            self.w_expand = torch.cat([key.view(-1, self.rank + self.rot), value], dim=0).contiguous()
        if self.sink:
            self.sink_values = tensors[self.sink_name].contiguous()

    def forward(self, ctx, x: torch.Tensor, cache: LayerCache, state=None) -> torch.Tensor:
        H, T = self.heads, x.shape[0]
        proj = ops.linear(x, self.w_in)
        cos, sin = self.position.tables(ctx)
        table = ctx.block_tables[cache.group]
        first = proj[:, :self._n_first]
        latent = proj[:, self._lat_col:self._lat_col + self.rank + self.rot] if self.own_rows else None

        def prepare(q, lat, query_latent, out=None):
            ops.latent_prepare_parts(q, lat, query_latent, cache.k_pages, self.norm_weight,
                                     self.query_norm_weight, cos, sin, ctx.positions, ctx.seq_of_token,
                                     table, H, self.nope, self.rot, self.rank, cache.page_size, self.eps,
                                     write_cache=cache.write and self.own_rows, pairing=self.pairing,
                                     query_latent_out=out)

        if self.q_rank:
            # the query latent normed into rows of its own (the product that follows wants
            # contiguous rows), the latent rows stored
            cq = torch.empty((T, self.q_rank), dtype=proj.dtype, device=proj.device)
            prepare(None, latent, first, cq)
            q = ops.linear(cq, self.w_uq)
            prepare(q, None, None)
        else:
            q = first
            prepare(q, latent, None)
        kd = self.nope + self.rot
        if self.w_expand is not None and q.dtype == torch.bfloat16 and q.stride(0) % 8 == 0 and q.data_ptr() % 16 == 0 \
                and ops.latent_expand_supported(q.dtype, H, kd, self.vdim, self.rank, self.rot, cache.page_size):
            pages = ops.latent_expand_pages(ctx, H, kd, self.vdim, self.rank, self.rot, cache.page_size, self.window)
            if pages:
                gate = proj[:, self._gate_col:self._gate_col + self._gate_rows] if self.gate else None
                options = ops.AttentionOptions(sink_values=self.sink_values, gate=gate, gate_wide=self.gate == "wide")
                return ops.linear(ops.latent_attention_expanded(ctx, q, cache.k_pages, table, self.w_expand, pages, H, kd,
                                                                self.vdim, cache.page_size, self.scale, self.window,
                                                                options), self.w_o)
        q = q.view(T, H, self.nope + self.rot) if q.is_contiguous() else \
            q.unflatten(1, (H, self.nope + self.rot))
        q_lat = ops.head_gemm(q[:, :, :self.nope], self.w_uk_t)
        o_lat = ops.latent_attention(ctx, q_lat, q[:, :, self.nope:], cache.k_pages, table,
                                     self.rank, self.rot, cache.page_size, self.scale, self.window,
                                     self.sink_values)
        o = ops.head_gemm(o_lat, self.w_uv)
        if self.gate:          # the gate's launch also lays the heads side by side, whatever the product's strides
            o = ops.gate_heads(o, proj[:, self._gate_col:self._gate_col + self._gate_rows], self.gate == "head")
        else:
            o = o.reshape(T, H * self.vdim)
        return ops.linear(o, self.w_o)


register_part("mixer", "latent_attention", LatentAttention)
