"""Typed configuration of the Gisodra design, read from ``config.json``.

The file lists the layers one by one; every entry names its mixer by ``type`` (``attention``:
grouped-query attention with biases, an RMS norm per query and key head, a window and a learned
sink, and optionally the keys and values of ANOTHER layer, ``kv_from``; ``gla``: gated linear
attention with a decay per key channel; ``latent_attention``: attention over a low-rank latent with
a window, a learned sink and a gate per head) with the mixer's sizes, and its feed-forward (dense,
or null for none).  Two models of the design may differ in every size, in the order of the layers
and in every constant; nothing here has a default that stands for a value of some particular
model.  What the file leaves out of an optional piece (a window, the cap on the logits, a layer's
feed-forward) is absent.  Sizes that the file does not give are read off the checkpoint's tensor
shapes.
"""
from __future__ import annotations

from dataclasses import dataclass, replace
from typing import Any, Dict, Optional, Tuple, Union

from .model_config import ConfigError
from .zokelix_config import RotaryConfig, _need


@dataclass(frozen=True)
class WindowSinkAttentionConfig:
    """``attention``."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    window: Optional[int]     # None: every earlier token
    kv_from: Optional[int]    # the layer whose keys and values this one reads; None: its own


@dataclass(frozen=True)
class ChannelDecayConfig:
    """``gla``."""
    heads: int
    dim: int
    vdim: int
    tau: float
    decay_rank: Optional[int]   # None until read off the checkpoint's 'a1'


@dataclass(frozen=True)
class WindowLatentConfig:
    """``latent_attention``."""
    heads: int
    dim: int                  # unrotated query/key values per head
    rot_dim: int              # rotated query/key values per head (the key part is shared)
    vdim: int
    kv_rank: int
    q_rank: Optional[int]     # None until read off the checkpoint's 'dq'
    scale: float
    rot: RotaryConfig
    window: Optional[int]


@dataclass(frozen=True)
class DenseFfnConfig:
    ff: int


MixerConfig = Union[WindowSinkAttentionConfig, ChannelDecayConfig, WindowLatentConfig]


@dataclass(frozen=True)
class GisodraLayer:
    type: str
    mixer: MixerConfig
    mlp: Optional[DenseFfnConfig]


@dataclass(frozen=True)
class GisodraConfig:
    architecture: str
    vocab_size: int
    width: int
    norm_eps: float
    logit_softcap: Optional[float]
    layers: Tuple[GisodraLayer, ...]
    eos_token_ids: Tuple[int, ...] = ()

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def max_position_embeddings(self) -> int:
        """No part of the design bounds a request's length."""
        return 1 << 30

    def cache_window(self, i: int) -> Optional[int]:
        """Tokens whose keys and values layer ``i`` has to keep: the widest window among the layers
        that attend them (None: all)."""
        windows = [x.mixer.window for j, x in enumerate(self.layers)
                   if isinstance(x.mixer, WindowSinkAttentionConfig) and (j == i or x.mixer.kv_from == i)]
        return None if None in windows else max(windows)

    @classmethod
    def from_json(cls, cfg: Dict[str, Any]) -> "GisodraConfig":
        vocab = _need(cfg, "vocab", "the file")
        width = _need(cfg, "width", "the file")
        eps = _need(cfg.get("norm"), "eps", "norm", float)
        cap = _need(cfg, "logit_softcap", "the file", float) if cfg.get("logit_softcap") is not None else None
        if cap is not None and not cap > 0:
            raise ConfigError(f"config.json: logit_softcap must be positive, got {cap}")
        layers = cfg.get("layers")
        if not isinstance(layers, list) or not layers:
            raise ConfigError("config.json: 'layers' must be a non-empty list")
        out = []
        for i, layer in enumerate(layers):
            where = f"layers[{i}]"
            kind = layer.get("type") if isinstance(layer, dict) else None
            reader = _MIXERS.get(kind)
            if reader is None:
                raise ConfigError(f"config.json: {where}.type {kind!r} is not supported "
                                  f"({', '.join(sorted(_MIXERS))})")
            out.append(GisodraLayer(kind, reader(layer.get("mixer"), where + ".mixer"),
                                    _mlp(layer.get("mlp"), where + ".mlp")))
        for i in range(len(out)):
            _check_source(out, i)
        eos = cfg.get("eos_token_id")
        eos_ids = () if eos is None else tuple(int(e) for e in (eos if isinstance(eos, (list, tuple)) else [eos]))
        return cls(architecture=str(cfg.get("architecture", "Gisodra")), vocab_size=vocab, width=width, norm_eps=eps,
                   logit_softcap=cap, layers=tuple(out), eos_token_ids=eos_ids)


def _check_source(layers, i: int) -> None:
    """A layer that reads another layer's keys and values: that layer comes earlier, has keys and
    values of its own, and heads of the same sizes."""
    mx = layers[i].mixer
    src_index = getattr(mx, "kv_from", None)
    if src_index is None:
        return
    where = f"config.json: layers[{i}].mixer.kv_from {src_index}"
    if not 0 <= src_index < i:
        raise ConfigError(f"{where} must name an earlier layer")
    src = layers[src_index].mixer
    if not isinstance(src, WindowSinkAttentionConfig) or src.kv_from is not None:
        raise ConfigError(f"{where} must name an attention layer with keys and values of its own")
    if (src.kv_heads, src.dim, src.vdim) != (mx.kv_heads, mx.dim, mx.vdim):
        raise ConfigError(f"{where}: that layer's kv_heads, dim or vdim differ from this layer's")


def _window(mx, where) -> Optional[int]:
    mask = mx.get("mask")
    return None if mask is None else _need(mask, "size", where + ".mask")


def _optional(mx, key, where):
    return _need(mx, key, where) if mx.get(key) is not None else None


def _own_rows_only(mx, where) -> None:
    if isinstance(mx, dict) and mx.get("kv_from") is not None:
        raise ConfigError(f"config.json: {where}.kv_from goes with the type attention only")


def _attention(mx, where) -> WindowSinkAttentionConfig:
    heads, kv_heads = _need(mx, "heads", where), _need(mx, "kv_heads", where)
    if heads % kv_heads:
        raise ConfigError(f"config.json: {where}.kv_heads {kv_heads} must divide heads {heads}")
    src = mx.get("kv_from")
    if src is not None and (not isinstance(src, int) or isinstance(src, bool) or src < 0):
        raise ConfigError(f"config.json: {where}.kv_from must be a layer's index, got {src!r}")
    return WindowSinkAttentionConfig(heads, kv_heads, _need(mx, "dim", where), _need(mx, "vdim", where),
                                     _need(mx, "scale", where, float), _window(mx, where), src)


def _gla(mx, where) -> ChannelDecayConfig:
    _own_rows_only(mx, where)
    tau = _need(mx, "tau", where, float)
    if not tau > 0:
        raise ConfigError(f"config.json: {where}.tau must be positive, got {tau}")
    return ChannelDecayConfig(_need(mx, "heads", where), _need(mx, "dim", where), _need(mx, "vdim", where), tau,
                              _optional(mx, "decay_rank", where))


def _latent(mx, where) -> WindowLatentConfig:
    _own_rows_only(mx, where)
    rot_dim = _need(mx, "rot_dim", where)
    rot = mx.get("rot")
    dims = _need(rot, "dims", where + ".rot")
    if dims % 2 or dims > rot_dim:
        raise ConfigError(f"config.json: {where}.rot.dims {dims} must be even and at most {rot_dim}")
    return WindowLatentConfig(
        heads=_need(mx, "heads", where), dim=_need(mx, "dim", where), rot_dim=rot_dim,
        vdim=_need(mx, "vdim", where), kv_rank=_need(mx, "kv_rank", where), q_rank=_optional(mx, "q_rank", where),
        scale=_need(mx, "scale", where, float),
        rot=RotaryConfig(_need(rot, "base", where + ".rot", float), dims, None), window=_window(mx, where))


_MIXERS = {"attention": _attention, "gla": _gla, "latent_attention": _latent}


def _mlp(ml, where) -> Optional[DenseFfnConfig]:
    if ml is None:
        return None
    kind = ml.get("kind") if isinstance(ml, dict) else None
    if kind != "dense":
        raise ConfigError(f"config.json: {where}.kind {kind!r} is not supported (dense)")
    return DenseFfnConfig(_need(ml, "ff", where))


def fill_from_tensor_shapes(cfg: GisodraConfig, shapes: Dict[str, Tuple[int, ...]]) -> GisodraConfig:
    """Sizes the file leaves to the checkpoint's tensor shapes: the rank of a decay's projection
    (``l<i>.mix.a1`` is [decay_rank, width]) and of a query latent (``l<i>.mix.dq`` is [q_rank, width])."""
    layers = list(cfg.layers)
    for i, layer in enumerate(layers):
        for kind, field, tensor in ((ChannelDecayConfig, "decay_rank", "a1"), (WindowLatentConfig, "q_rank", "dq")):
            if isinstance(layer.mixer, kind) and getattr(layer.mixer, field) is None:
                shape = shapes.get(f"l{i}.mix.{tensor}")
                if shape is None or len(shape) != 2:
                    raise ConfigError(f"config.json: layers[{i}].mixer has no '{field}' and the checkpoint no "
                                      f"matrix 'l{i}.mix.{tensor}'")
                layers[i] = replace(layer, mixer=replace(layer.mixer, **{field: int(shape[0])}))
    return replace(cfg, layers=tuple(layers))
