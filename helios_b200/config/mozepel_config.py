"""Typed configuration of the Mozepel design, read from ``config.json``.

The file lists the layers one by one; every entry names its mixer by ``type`` (``retention``:
linear attention with a fixed decay a head, rotated queries and keys and a norm per head;
``parallel``: two mixers side by side on the same input, ``left`` window attention that sees
older tokens as means of whole blocks, ``right`` linear attention with a fixed decay a head on
activated projections) with the mixer's sizes, and its feed-forward (dense, or null for none).
An entry with ``weights_of`` runs the tensors of the layer it names with a cache and a state
of its own.  Two models of the design may differ in every size, in the order of the layers
and in every constant; nothing here has a default that stands for a value of some particular
model.  What the file leaves out of an optional piece (a rotary scaling, the short
convolution, the pooled blocks, a layer's feed-forward) is absent.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Any, Dict, Optional, Tuple, Union

from .model_config import ConfigError, RopeScaling
from .zokelix_config import _need


@dataclass(frozen=True)
class RotationConfig:
    base: float
    dims: int
    scaling: Optional[RopeScaling]


@dataclass(frozen=True)
class RetentionConfig:
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]
    rot: RotationConfig


@dataclass(frozen=True)
class PooledWindowConfig:
    """``left`` of ``parallel``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    conv: int                 # taps of the short convolution on q, k and v; 0: none
    rot: RotationConfig
    window: int
    pool: int                 # tokens a block; 0: tokens behind the window are not seen at all


@dataclass(frozen=True)
class DecayedLinearConfig:
    """``right`` of ``parallel``."""
    heads: int
    dim: int
    vdim: int
    decay: Tuple[float, ...]


@dataclass(frozen=True)
class SideBySideConfig:
    left: PooledWindowConfig
    left_scale: float
    right: DecayedLinearConfig
    right_scale: float


@dataclass(frozen=True)
class DenseFfnConfig:
    ff: int


MixerConfig = Union[RetentionConfig, SideBySideConfig]


@dataclass(frozen=True)
class MozepelLayer:
    type: str
    mixer: MixerConfig
    mlp: Optional[DenseFfnConfig]
    weights_of: int           # the layer whose tensors this entry runs (its own index: its own)


@dataclass(frozen=True)
class MozepelConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    residual_factor: float    # on the stream, where a sublayer's output joins it
    layers: Tuple[MozepelLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        """No part of the design bounds a request's length."""
        return 1 << 30

    @classmethod
    def from_json(cls, cfg: Dict[str, Any]) -> "MozepelConfig":
        vocab = _need(cfg, "vocab", "the file")
        width = _need(cfg, "width", "the file")
        eps = _need(cfg.get("norm"), "eps", "norm", float)
        alpha = _need(cfg, "postln_alpha", "the file", float)
        entries = cfg.get("layers")
        if not isinstance(entries, list) or not entries:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out = []
        for i, entry in enumerate(entries):
            where = f"layers[{i}]"
            if not isinstance(entry, dict):
                raise ConfigError(f"config.json: {where} must be an object")
            src = _source(entries, i)
            own = entries[src]
            for key in ("type", "mixer", "mlp"):
                if src != i and key in entry and entry[key] != own.get(key):
                    raise ConfigError(f"config.json: {where} runs the tensors of layer {src} but differs from "
                                      f"it in '{key}'")
            kind = own.get("type")
            reader = _MIXERS.get(kind)
            if reader is None:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not supported "
                                  f"({', '.join(sorted(_MIXERS))})")
            out.append(MozepelLayer(kind, reader(own.get("mixer"), where + ".mixer"),
                                    _mlp(own.get("mlp"), where + ".mlp"), src))
        eos = cfg.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(architecture=str(cfg.get("architecture", "Mozepel")), vocab_size=vocab, width=width,
                   norm_eps=eps, residual_factor=alpha, layers=tuple(out), eos_token_ids=eos_ids)


def _source(entries, i: int) -> int:
    """The layer whose tensors entry ``i`` runs, through entries that point on."""
    seen, j = {i}, i
    while isinstance(entries[j], dict) and entries[j].get("weights_of") is not None:
        to = entries[j]["weights_of"]
        if not isinstance(to, int) or isinstance(to, bool) or not 0 <= to < len(entries) or to in seen:
            raise ConfigError(f"config.json: layers[{j}].weights_of {to!r} must name a layer with tensors")
        seen.add(to)
        j = to
    return j


def _rotation(rot, where, most: int) -> RotationConfig:
    dims = _need(rot, "dims", where)
    if dims % 2 or dims > most:
        raise ConfigError(f"config.json: {where}.dims {dims} must be even and at most {most}")
    sc = rot.get("scaling")
    scaling = None
    if sc:
        at = where + ".scaling"
        scaling = RopeScaling(factor=_need(sc, "factor", at, float), low_freq_factor=_need(sc, "low", at, float),
                              high_freq_factor=_need(sc, "high", at, float),
                              original_max_position_embeddings=_need(sc, "original", at, float))
        if scaling.high_freq_factor <= scaling.low_freq_factor:
            raise ConfigError(f"config.json: {at}.high must exceed low")
    return RotationConfig(_need(rot, "base", where, float), dims, scaling)


def _decay(mx, heads: int, where) -> Tuple[float, ...]:
    v = mx.get("decay")
    if not isinstance(v, (list, tuple)) or len(v) != heads \
            or any(isinstance(d, bool) or not isinstance(d, (int, float)) for d in v):
        raise ConfigError(f"config.json: {where}.decay must list {heads} numbers, one a head")
    if any(not 0.0 <= float(d) <= 1.0 for d in v):
        raise ConfigError(f"config.json: {where}.decay must lie between 0 and 1")
    return tuple(float(d) for d in v)


def _retention(mx, where) -> RetentionConfig:
    heads, dim = _need(mx, "heads", where), _need(mx, "dim", where)
    return RetentionConfig(heads, dim, _need(mx, "vdim", where), _decay(mx, heads, where),
                           _rotation(mx.get("rot"), where + ".rot", dim))


def _optional(d, key, where) -> int:
    """A positive integer, or 0 where the file has none."""
    return _need(d, key, where) if isinstance(d, dict) and d.get(key) else 0


def _side_by_side(mx, where) -> SideBySideConfig:
    ls, rs = _need(mx, "left_scale", where, float), _need(mx, "right_scale", where, float)
    le, at = mx.get("left"), where + ".left"
    heads, kv_heads = _need(le, "heads", at), _need(le, "kv_heads", at)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {at}.kv_heads {kv_heads} must divide heads {heads}")
    dim = _need(le, "dim", at)
    mask = le.get("mask")
    left = PooledWindowConfig(heads, kv_heads, dim, _need(le, "vdim", at), _need(le, "scale", at, float),
                              _optional(le, "conv", at), _rotation(le.get("rot"), at + ".rot", dim),
                              _need(mask, "size", at + ".mask"), _optional(mask, "pool", at + ".mask"))
    ri, at = mx.get("right"), where + ".right"
    rheads = _need(ri, "heads", at)
    right = DecayedLinearConfig(rheads, _need(ri, "dim", at), _need(ri, "vdim", at), _decay(ri, rheads, at))
    return SideBySideConfig(left, ls, right, rs)


_MIXERS = {"retention": _retention, "parallel": _side_by_side}


def _mlp(ml, where) -> Optional[DenseFfnConfig]:
    if ml is None:
        return None
    kind = ml.get("kind") if isinstance(ml, dict) else None
    if kind != "dense":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not supported (dense)")
    return DenseFfnConfig(_need(ml, "ff", where))
