"""Plan of the Mozepel design: token embedding; blocks that norm the SUM of the weighted stream
and a sublayer's output, norm(a x + mixer(x)) and norm(a x + ff(x)), so that the sublayers read
the normed stream itself; two kinds of mixer, chosen layer by layer — linear attention with a
fixed decay a head, rotated queries and keys, a norm per head and a silu gate; and, side by
side on the same input, window attention that sees older tokens as means of whole blocks
(short convolutions, weighted q/k norm, rotation with stretched long waves) and linear
attention with a fixed decay a head on activated projections (one norm over the row, a
sigmoid gate) — and a gated dense feed-forward or none; a final RMS norm and an output head
of its own.

A layer may be run several times: an entry that names another layer's tensors becomes one
more run of that layer in the schedule, with a cache and a state of its own.
"""
from __future__ import annotations

from ..config.mozepel_config import (DecayedLinearConfig, MozepelConfig, PooledWindowConfig, RetentionConfig,
                                     RotationConfig, SideBySideConfig)
from ..config.registry import register_architecture
from ..parts import ModelPlan, OutputHead, Run, TokenEmbedding, part_class


def build_mozepel_plan(cfg: MozepelConfig) -> ModelPlan:
    norm_cls = part_class("norm", "rmsnorm")
    block_cls = part_class("block", "normed_sum")
    decay_cls = part_class("mixer", "fixed_decay")
    window_cls = part_class("mixer", "pooled_window")
    pair_cls = part_class("mixer", "side_by_side")
    ffn_cls = part_class("feed_forward", "gated_mlp")
    rotary_cls = part_class("position_encoding", "rotary")
    encodings = {}          # one encoding per distinct rotation: layers that agree share its tables

    def norm():
        return norm_cls(cfg.width, cfg.norm_eps, tensor_name="")

    def encoding(rot: RotationConfig):
        if rot not in encodings:
            encodings[rot] = rotary_cls(rot.dims, rot.base, rot.scaling)
        return encodings[rot]

    def retention(mx: RetentionConfig):
        return decay_cls(cfg.width, mx.heads, mx.dim, mx.vdim, mx.decay, cfg.norm_eps, key_scale=mx.dim ** -0.5,
                         position=encoding(mx.rot), rotary_dim=mx.rot.dims, norm="head", gate="silu")

    def window(mx: PooledWindowConfig):
        return window_cls(cfg.width, mx.heads, mx.kv_heads, mx.dim, mx.vdim, mx.scale, mx.window, mx.pool,
                          cfg.norm_eps, encoding(mx.rot), mx.rot.dims, taps=mx.conv)

    def decayed(mx: DecayedLinearConfig):
        return decay_cls(cfg.width, mx.heads, mx.dim, mx.vdim, mx.decay, cfg.norm_eps, activation="silu",
                         norm="row", gate="sigmoid")

    def mixer(mx):
        if isinstance(mx, RetentionConfig):
            return retention(mx)
        if isinstance(mx, SideBySideConfig):
            return pair_cls(window(mx.left), decayed(mx.right), mx.left_scale, mx.right_scale)
        raise ValueError(f"no mixer for {type(mx).__name__}")

    layers, prefixes, index = [], [], {}
    for i, layer in enumerate(cfg.layers):
        if layer.weights_of != i:
            continue
        ffn = ffn_cls(cfg.width, layer.mlp.ff, "silu", names=("gate", "up", "down")) if layer.mlp else None
        index[i] = len(layers)
        layers.append(block_cls(mixer(layer.mixer), norm(), ffn, norm() if ffn is not None else None,
                                factor=cfg.residual_factor))
        prefixes.append(f"l{i}.")
    return ModelPlan(
        config=cfg,
        embedding=TokenEmbedding(cfg.vocab_size, cfg.width, tensor_name=""),
        position=None,
        layers=layers,
        layer_prefixes=prefixes,
        final_norm=norm(),
        head=OutputHead(cfg.vocab_size, cfg.width, tensor_name=""),
        schedule=[Run(index[layer.weights_of]) for layer in cfg.layers],
        embedding_prefix="embed",
        final_norm_prefix="final.norm",
        head_prefix="head",
        benign_suffixes=(),
    )


def _toy_config(sizes):
    """config.json of a small model of the design from the sizes ``make-toy-model`` takes: two
    retention layers, then two mixers side by side, in turn; the last layer runs the first
    layer's tensors once more when there are four or more."""
    width = sizes["hidden_size"]
    heads = sizes["heads"]
    hd = sizes.get("head_dim") or max(8, (width // heads) // 2 * 2)
    inner = sizes.get("intermediate_size") or 2 * width
    n = sizes["layers"]
    decay = [1.0 - 2.0 ** -(3 + h % 6) for h in range(heads)]
    layers = []
    for i in range(n):
        if i % 3 == 2:
            entry = {"type": "parallel", "mixer": {
                "left": {"heads": heads, "kv_heads": sizes["kv_heads"], "dim": hd, "vdim": hd, "scale": hd ** -0.5,
                         "conv": 4, "rot": {"dims": hd, "base": 10000.0}, "mask": {"size": 48, "pool": 8}},
                "left_scale": 0.7, "right": {"heads": heads, "dim": hd, "vdim": hd, "decay": decay},
                "right_scale": 0.4}}
        else:
            entry = {"type": "retention", "mixer": {"heads": heads, "dim": hd, "vdim": hd, "decay": decay,
                                                    "rot": {"dims": hd, "base": 10000.0}}}
        layers.append({**entry, "mlp": {"kind": "dense", "ff": inner}})
    if n >= 4:
        layers[-1] = {**layers[0], "weights_of": 0}
    return {"architecture": "Mozepel", "vocab": sizes["vocab_size"], "width": width,
            "norm": {"eps": sizes["rms_eps"]}, "postln_alpha": 1.5, "layers": layers}


register_architecture("Mozepel", MozepelConfig.from_json, build_mozepel_plan, toy_config=_toy_config, replace=True)
