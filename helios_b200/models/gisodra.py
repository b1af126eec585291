"""Plan of the Gisodra design: token embedding; blocks with a norm before AND after each sublayer,
x + norm(mixer(norm(x))) and x + norm(ff(norm(x))); three kinds of mixer, chosen layer by layer —
grouped-query window attention without positions, with biases, a weighted norm per query and key
head and a learned sink, optionally on the keys and values that another layer keeps; gated linear
attention with a decay per key channel; window attention over a low-rank latent whose queries pass
a latent of their own, with rotary positions on halves of a shared key part, a learned sink and a
gate per head — and a gated dense feed-forward (tanh form of gelu) or none; a final RMS norm, the
embedding table as output head, and a cap on the logits.

Every layer's parts are made from that layer's entry of the configuration, so the order of the
layers and all sizes are the file's.  Layers with equal rotary constants share one encoding.  A
layer that reads another layer's keys and values is scheduled with that layer's cache and does not
write it; the pages keep as many tokens as the widest of the windows on them wants.
"""
from __future__ import annotations

from ..config.gisodra_config import (ChannelDecayConfig, GisodraConfig, WindowLatentConfig,
                                     WindowSinkAttentionConfig, fill_from_tensor_shapes)
from ..config.registry import register_architecture
from ..parts import ModelPlan, OutputHead, TokenEmbedding, part_class
from ..parts.plan import Run
from .zokelix import _encoding


def build_gisodra_plan(cfg: GisodraConfig) -> ModelPlan:
    norm_cls = part_class("norm", "rmsnorm")
    block_cls = part_class("block", "sandwich")
    ffn_cls = part_class("feed_forward", "gated_mlp")
    encodings = {}          # one encoding per distinct set of rotary constants

    def norm():
        return norm_cls(cfg.width, cfg.norm_eps, tensor_name="")

    def mixer(i, mx):
        if isinstance(mx, WindowSinkAttentionConfig):
            own = mx.kv_from is None
            return part_class("mixer", "sink_gqa_attention")(
                cfg.width, mx.heads, mx.kv_heads, mx.dim, mx.scale, value_dim=mx.vdim, qk_norm=True,
                eps=cfg.norm_eps, sink="learned", head_gate=False, window=mx.window, qk_bias=True, own_keys=own,
                cache_window=cfg.cache_window(i) if own else -1)
        if isinstance(mx, ChannelDecayConfig):
            if mx.decay_rank is None:
                raise ValueError(f"layer {i}: the rank of the decay's projection is neither in config.json "
                                 "('decay_rank') nor read off a checkpoint")
            return part_class("mixer", "channel_decay")(
                cfg.width, mx.heads, mx.dim, mx.vdim, mx.decay_rank, mx.tau, cfg.norm_eps, q_scale=mx.dim ** -0.5)
        if isinstance(mx, WindowLatentConfig):
            if mx.q_rank is None:
                raise ValueError(f"layer {i}: the rank of the query latent is neither in config.json "
                                 "('q_rank') nor read off a checkpoint")
            return part_class("mixer", "latent_attention")(
                cfg.width, mx.heads, mx.dim, mx.rot_dim, mx.vdim, mx.kv_rank, mx.scale, cfg.norm_eps,
                _encoding(mx.rot, encodings), q_rank=mx.q_rank, pairing="halves", gate="head", window=mx.window,
                sink=True)
        raise ValueError(f"layer {i}: no mixer for {type(mx).__name__}")

    layers, prefixes, schedule = [], [], []
    for i, layer in enumerate(cfg.layers):
        ffn = (norm(), ffn_cls(cfg.width, layer.mlp.ff, "gelu_tanh", names=("gate", "up", "down")), norm()) \
            if layer.mlp is not None else ()
        layers.append(block_cls(norm(), mixer(i, layer.mixer), norm(), *ffn))
        prefixes.append(f"l{i}.")
        src = getattr(layer.mixer, "kv_from", None)
        schedule.append(Run(i) if src is None else Run(i, cache=src, writes_cache=False))   # one run a layer
    return ModelPlan(
        config=cfg,
        embedding=TokenEmbedding(cfg.vocab_size, cfg.width, tensor_name=""),
        position=None,
        layers=layers,
        layer_prefixes=prefixes,
        final_norm=norm(),
        head=OutputHead(cfg.vocab_size, cfg.width, tensor_name="", softcap=cfg.logit_softcap),
        schedule=schedule,
        embedding_prefix="embed",
        final_norm_prefix="final.norm",
        head_prefix="head",
        tied={"head": "embed"},
        benign_suffixes=(),
    )


def _toy_config(sizes):
    """config.json of a small model of the design from the sizes ``make-toy-model`` takes: the kinds of
    mixer in turn (latent attention, attention, gated linear attention, attention on the keys and
    values of the attention layer before); gated linear attention has no feed-forward."""
    width = sizes["hidden_size"]
    heads = sizes["heads"]
    hd = sizes.get("head_dim") or max(8, (width // heads) // 2 * 2)
    inner = sizes.get("intermediate_size") or 2 * width
    layers = []
    for i in range(sizes["layers"]):
        kind = ("latent_attention", "attention", "gla", "attention")[i % 4]
        if kind == "latent_attention":
            rot = max(2, hd // 2 // 2 * 2)
            mixer = {"heads": heads, "dim": hd, "rot_dim": rot, "vdim": hd, "kv_rank": 2 * hd,
                     "q_rank": max(8, width // 4), "scale": (hd + rot) ** -0.5, "mask": {"size": 32},
                     "rot": {"base": sizes["rope_theta"], "dims": rot}}
        elif kind == "attention":
            mixer = {"heads": heads, "kv_heads": sizes["kv_heads"], "dim": hd, "vdim": hd, "scale": hd ** -0.5,
                     "mask": {"size": 48}}
            if i % 4 == 3:
                mixer["kv_from"] = i - 2
        else:
            mixer = {"heads": heads, "dim": hd, "vdim": hd, "tau": 16.0, "decay_rank": 16}
        layers.append({"type": kind, "mixer": mixer, "mlp": None if kind == "gla" else {"kind": "dense", "ff": inner}})
    return {"architecture": "Gisodra", "vocab": sizes["vocab_size"], "width": width,
            "norm": {"eps": sizes["rms_eps"]}, "logit_softcap": 30.0, "layers": layers}


register_architecture("Gisodra", GisodraConfig.from_json, build_gisodra_plan, toy_config=_toy_config,
                      sizes_from_tensors=fill_from_tensor_shapes, replace=True)
