"""The Gisodra design against a plain float64 implementation (``plain_gisodra``): every mechanism
alone on made inputs, then whole models of several shapes through the step function (whole
prompts, decoding, portions, mixed batches, replay, generation), and models drawn at random."""
from __future__ import annotations

import json
import math
import random
from types import SimpleNamespace

import pytest
import torch

import plain_gisodra as pg
import trace_util as tu
from conftest import F32_ATOL, random_tokens, read_folder

DTYPES = ["float32", "bfloat16"]


# ---------------------------------------------------------------------- configurations
def _att(heads, kv, dim, vdim, scale, window, kv_from=None):
    mx = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale}
    if window is not None:
        mx["mask"] = {"size": window}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "attention", "mixer": mx}


def _gla(heads, dim, vdim, tau, rank):
    return {"type": "gla", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau, "decay_rank": rank}}


def _lat(heads, dim, rot_dim, vdim, rank, q_rank, scale, base, window):
    mx = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank,
          "scale": scale, "rot": {"dims": rot_dim, "base": base}}
    if window is not None:
        mx["mask"] = {"size": window}
    return {"type": "latent_attention", "mixer": mx}


def _model(vocab, width, eps, cap, layers):
    cfg = {"architecture": "Gisodra", "vocab": vocab, "width": width, "norm": {"eps": eps},
           "layers": [dict(layer, mlp=None if ff is None else {"kind": "dense", "ff": ff}) for layer, ff in layers]}
    if cap is not None:
        cfg["logit_softcap"] = cap
    return cfg


# heads of 32 with values of 32 (the tensor-core kernels' smallest) and a latent of 64 + 16 (the
# tensor-core latent kernel); the reader of another layer's keys has a WIDER window than their owner,
# another one reads the same keys through a narrower one
GS_A = _model(211, 96, 1e-5, 4.0, [
    (_lat(4, 32, 16, 32, 64, 40, 0.15, 10000.0, 24), 80),
    (_att(4, 2, 32, 32, 0.2, 40), 80),
    (_gla(3, 16, 24, 8.0, 8), None),
    (_att(4, 2, 32, 32, 0.18, 57, kv_from=1), 48),
    (_lat(2, 16, 16, 48, 64, 24, 0.2, 500.0, 70), None),
    (_att(4, 2, 32, 32, 0.18, 9, kv_from=1), 80),
])
# a width that is no multiple of 8, heads of 10 and 7, values wider than keys, a latent of 20 + 6, a
# window of one token, one attention layer without a window, a decay without root (tau 1) and of a
# rank that is no multiple of 4, no cap, the reader right after its source
GS_B = _model(131, 50, 2e-6, None, [
    (_gla(2, 7, 5, 1.0, 3), 30),
    (_att(3, 3, 10, 14, 0.4, 7), None),
    (_att(3, 3, 10, 14, 0.3, 1, kv_from=1), 20),
    (_lat(2, 10, 6, 12, 20, 7, 0.3, 77.0, 1), 30),
    (_att(5, 1, 10, 6, 0.3, None), None),
    (_lat(3, 8, 4, 6, 12, 9, 0.35, 77.0, 33), 24),
])
# values of another size than keys on the tensor cores, a recurrence with heads of 64 x 128 and one of
# 128 x 32, a latent of 128 + 32, windows beyond a tile of 128 keys
GS_C = _model(180, 128, 1e-5, 2.5, [
    (_gla(4, 64, 128, 16.0, 16), 96),
    (_att(8, 2, 96, 64, 0.1, 100), 64),
    (_lat(4, 64, 32, 64, 128, 96, 0.1, 5000.0, 130), 64),
    (_att(8, 2, 96, 64, 0.12, 150, kv_from=1), None),
    (_gla(2, 128, 32, 2.0, 20), 64),
])
GS_CONFIGS = {"gs_a": GS_A, "gs_b": GS_B, "gs_c": GS_C}
GS_SEEDS = {"gs_a": 3, "gs_b": 4, "gs_c": 5}
GS_ALONE = {
    "attention_only": _model(97, 64, 1e-5, 3.0, [(_att(4, 2, 16, 24, 0.3, 12), None)]),
    "borrowed_keys": _model(97, 64, 1e-5, None, [(_att(4, 2, 24, 16, 0.3, 5), None),
                                                 (_att(4, 2, 24, 16, 0.3, 21, kv_from=0), None)]),
    "gla_only": _model(97, 64, 1e-5, 3.0, [(_gla(2, 24, 40, 4.0, 12), None)]),
    "latent_only": _model(97, 64, 1e-5, 3.0, [(_lat(4, 16, 8, 16, 32, 24, 0.3, 1000.0, 19), None)]),
    "feed_forward": _model(97, 64, 1e-5, 3.0, [(_gla(2, 8, 16, 4.0, 4), 72)]),
}


def _lively(cfg, weights, spread=2.0):
    """Random matrices of a small scale give nearly flat attention, decays that hardly depend on the
    token and logits near 0, under which a wrong key, state or cap would hide.  Scale what the scores
    grow with so that a query's scores spread by about ``spread``, the decay's matrices, the gates and
    the embedding (whose rows are the output head's too).  The norms after the sublayers are scaled down,
    and the recurrence's keys lean towards its queries: a norm per head makes of a head whose q . k is
    near 0 (a request's first token) whatever rounding left of its sign."""
    w = {k: v.clone() for k, v in weights.items()}
    std, width = 0.02, cfg["width"]
    w["embed"] *= 5.0
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.mix.", layer["mixer"]
        for n in ("norm1b", "norm2b"):
            if f"l{i}.{n}" in w:
                w[f"l{i}.{n}"] *= 0.3
        if layer["type"] == "gla":
            w[p + "k"] = 0.7 * w[p + "k"] + 0.7 * w[p + "q"]
            w[p + "a1"] *= 1.0 / (std * math.sqrt(width))
            w[p + "a2"] *= 1.0 / (std * math.sqrt(mx["decay_rank"]))
            w[p + "a2.b"] += 1.0
            w[p + "g"] *= 8.0
            continue
        want = math.sqrt(spread / (mx["scale"] * math.sqrt(mx["dim"])))      # size of a q and of a k value
        if layer["type"] == "attention":
            w[p + "q.norm"] *= want
            if p + "k.norm" in w:
                w[p + "k.norm"] *= want
                w[p + "k.b"] *= 20.0
                w[p + "v.b"] *= 20.0
            w[p + "q.b"] *= 10.0
            w[p + "sink"] += 1.0
        else:
            w[p + "uq"] *= want / (std * math.sqrt(mx["q_rank"]))
            w[p + "uk"] *= want / (std * math.sqrt(mx["kv_rank"]))
            w[p + "g"] *= 20.0                       # gates away from one half
    return w


@pytest.fixture(scope="module")
def gs_folders(tmp_path_factory):
    """Model folders with random weights made lively; ``config.json`` is then written WITHOUT the
    ranks that a reader has to take from the tensors' shapes."""
    from safetensors.torch import save_file
    from helios_b200.weights import write_model_folder

    out = {}
    base = tmp_path_factory.mktemp("gisodra")
    for name, cfg in {**GS_CONFIGS, **GS_ALONE}.items():
        folder = write_model_folder(base / name, cfg, GS_SEEDS.get(name, 9))
        _cfg, weights = read_folder(folder)
        save_file(_lively(cfg, weights), str(folder / "model.safetensors"))
        _write_lean(folder, cfg)
        out[name] = folder
    return out


def _write_lean(folder, cfg):
    lean = json.loads(json.dumps(cfg))
    for layer in lean["layers"]:
        layer["mixer"].pop("q_rank", None)
        layer["mixer"].pop("decay_rank", None)
    (folder / "config.json").write_text(json.dumps(lean))


def _weights(weights, dtype):
    """What the engine computes with: matrices rounded to bfloat16 in bfloat16 mode."""
    return {k: (v.to(torch.bfloat16) if dtype == "bfloat16" and v.dim() >= 2 else v).double()
            for k, v in weights.items()}


def _plain(cfg, weights, dtype, requests):
    w = _weights(weights, dtype)
    return {rid: pg.forward(cfg, w, toks)[0] for rid, toks in requests.items()}


def _core(folder, dtype, max_tokens, page_size=16, max_slots=4, graphs=True):
    from helios_b200.engine.core import EngineCore
    from helios_b200.engine.model import DecoderModel

    model = DecoderModel.from_folder(folder, dtype=dtype)
    return EngineCore(model, page_size=page_size, num_pages=-(-max_tokens // page_size),
                      max_slots=max_slots, poison_cache=float("nan"), use_cuda_graphs=graphs)


def _check(tb, got, plain, dtype, what, most=0.05, outliers=0.0):
    """Every wanted row against the plain model: float32 value by value, relative to the row's largest
    (at least 1); bfloat16 by the root mean
    square over the vocabulary, relative to the row's: no more than a share ``outliers`` of the rows
    above ``most`` and half of them below 2 % (what 16-bit activations leave; a norm per head makes of
    a sum near 0 whatever rounding left of it, so single rows of a model drawn at random may stand
    further off, where a wrong key or state would move most of them)."""
    assert set(got) == set(tb.rows), what
    rel, at = [], []
    for step, rows in tb.rows.items():
        want = torch.stack([plain[rid][pos] for rid, pos in rows])
        g = torch.from_numpy(got[step]).double()
        assert torch.isfinite(g).all(), (what, step)
        if dtype == "float32":
            err = (g - want).abs().amax(-1) / want.abs().amax(-1).clamp(min=1.0)
            assert float(err.max()) < F32_ATOL, (what, tb.steps[step], rows[int(err.argmax())], float(err.max()))
            continue
        rel += ((g - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()).tolist()
        at += rows
    if dtype == "float32":
        return
    rel = torch.tensor(rel)
    worst = int(rel.argmax())
    assert float(rel.median()) < 0.02 and float((rel > most).double().mean()) <= outliers, \
        f"{what}: median {float(rel.median()):.4f}, worst {float(rel[worst]):.4f} at (request, position) = {at[worst]}"


def _requests(cfg, lengths, seed):
    return {f"q{i}": random_tokens(cfg["vocab"], n, seed + i) for i, n in enumerate(lengths)}


def _dt(dtype):
    return torch.float32 if dtype == "float32" else torch.bfloat16


# ====================================================================== without a GPU
def test_configuration_is_read_layer_by_layer_and_faults_name_the_key():
    from helios_b200.config import ConfigError
    from helios_b200.config.gisodra_config import (ChannelDecayConfig, GisodraConfig, WindowLatentConfig,
                                                   WindowSinkAttentionConfig, fill_from_tensor_shapes)

    cfg = GisodraConfig.from_json(GS_A)
    assert [type(l.mixer) for l in cfg.layers] == [WindowLatentConfig, WindowSinkAttentionConfig, ChannelDecayConfig,
                                                   WindowSinkAttentionConfig, WindowLatentConfig,
                                                   WindowSinkAttentionConfig]
    assert cfg.logit_softcap == 4.0 and cfg.layers[2].mlp is None and cfg.layers[0].mlp.ff == 80
    assert cfg.layers[3].mixer.kv_from == 1 and cfg.layers[1].mixer.kv_from is None
    assert cfg.cache_window(1) == 57                      # the widest of the windows on layer 1's keys
    b = GisodraConfig.from_json(GS_B)
    assert b.logit_softcap is None and b.layers[4].mixer.window is None and b.cache_window(4) is None
    assert b.layers[0].mixer.tau == 1.0
    lean = json.loads(json.dumps(GS_A))
    del lean["layers"][2]["mixer"]["decay_rank"], lean["layers"][0]["mixer"]["q_rank"]
    got = GisodraConfig.from_json(lean)
    assert got.layers[2].mixer.decay_rank is None and got.layers[0].mixer.q_rank is None
    got = fill_from_tensor_shapes(got, {"l2.mix.a1": (8, 96), "l0.mix.dq": (40, 96)})
    assert got == cfg
    with pytest.raises(ConfigError, match="decay_rank"):
        fill_from_tensor_shapes(GisodraConfig.from_json(lean), {"l0.mix.dq": (40, 96)})
    for path, value, word in [(("layers", 0, "mixer", "rot", "dims"), 7, "dims"),
                              (("layers", 1, "mixer", "kv_heads"), 3, "kv_heads"),
                              (("layers", 1, "mixer", "mask", "size"), 0, "size"),
                              (("layers", 2, "mixer", "tau"), 0.0, "tau"),
                              (("layers", 2, "mixer", "tau"), None, "tau"),
                              (("layers", 2, "mixer", "kv_from"), 1, "kv_from"),
                              (("layers", 3, "mixer", "kv_from"), 3, "kv_from"),
                              (("layers", 3, "mixer", "kv_from"), 2, "kv_from"),
                              (("layers", 5, "mixer", "kv_from"), 3, "kv_from"),
                              (("layers", 3, "mixer", "vdim"), 16, "kv_from"),
                              (("layers", 0, "mixer", "scale"), None, "scale"),
                              (("layers", 0, "mlp", "kind"), "moe", "kind"),
                              (("layers", 0, "type"), "conv", "type"),
                              (("logit_softcap",), -1.0, "logit_softcap"),
                              (("norm",), {}, "eps")]:
        bad = json.loads(json.dumps(GS_A))
        at = bad
        for key in path[:-1]:
            at = at[key]
        if value is None:
            del at[path[-1]]
        else:
            at[path[-1]] = value
        with pytest.raises(ConfigError, match=word):
            GisodraConfig.from_json(bad)


def test_plan_names_every_tensor_and_sizes_caches_and_states():
    from helios_b200.cache.manager import cache_groups_of
    from helios_b200.config.gisodra_config import GisodraConfig
    from helios_b200.models import build_gisodra_plan
    from helios_b200.weights.loader import expected_tensors

    plan = build_gisodra_plan(GisodraConfig.from_json(GS_A))
    names = expected_tensors(plan)
    for name in ["embed", "final.norm", "l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "l0.mix.dq", "l0.mix.dq.norm",
                 "l0.mix.uq", "l0.mix.dkv", "l0.mix.dkv.norm", "l0.mix.uk", "l0.mix.uv", "l0.mix.sink", "l0.mix.g",
                 "l0.mix.o", "l0.mlp.gate", "l1.mix.q", "l1.mix.q.b", "l1.mix.k.b", "l1.mix.v.b", "l1.mix.q.norm",
                 "l1.mix.k.norm", "l1.mix.sink", "l2.mix.a1", "l2.mix.a2", "l2.mix.a2.b", "l2.mix.norm", "l2.mix.g",
                 "l3.mix.q.b", "l3.mix.q.norm", "l3.mix.sink"]:
        assert name in names, name
    for name in ["l1.mix.g", "l1.mix.o.b", "l2.norm2", "l2.norm2b", "l2.mlp.gate", "l2.mix.sink", "l3.mix.k", "l3.mix.v",
                 "l3.mix.k.b", "l3.mix.v.b", "l3.mix.k.norm", "l0.mix.q", "l0.mlp.gate.b"]:
        assert name not in names, name
    assert plan.tied == {"head": "embed"}
    assert names["l0.mix.g"][2].shape == (4, 96) and names["l2.mix.a2"][2].shape == (48, 8)
    assert names["l2.mix.norm"][2].shape == (24,) and names["l1.mix.q.norm"][2].shape == (32,)
    assert [(r.layer, r.cache, r.writes_cache) for r in plan.schedule] == \
        [(0, None, True), (1, None, True), (2, None, True), (3, 1, False), (4, None, True), (5, 1, False)]
    specs, where = cache_groups_of(plan)
    assert sorted(where) == [0, 1, 4]
    assert {(s.planes, s.num_kv_heads, s.head_dim, s.window) for s in specs} == {(1, 1, 80, 24), (2, 2, 32, 57),
                                                                                 (1, 1, 80, 70)}
    assert plan.layers[2].mixer.state_spec().shape == (3 * 16 * 24,)


def test_toy_model_of_the_design_from_the_command_line(tmp_path, capsys):
    from helios_b200 import cli

    assert cli.main(["make-toy-model", "--arch", "gisodra", "--out", str(tmp_path / "toy"), "--layers", "5",
                     "--hidden", "64", "--heads", "4", "--kv-heads", "2"]) == 0
    assert cli.main(["info", "--model", str(tmp_path / "toy")]) == 0
    text = capsys.readouterr().out
    assert "Gisodra" in text and "ChannelDecayMixer" in text and "SandwichBlock" in text


def test_the_plain_model_in_portions_is_the_plain_model():
    """The oracle itself: a prompt cut in three, with borrowed keys and a carried state."""
    from helios_b200.weights.random_init import random_tensors
    from helios_b200.config.registry import resolve_architecture

    arch = resolve_architecture(GS_B)
    w = {k: v.double() for k, v in random_tensors(arch.build_plan(arch.parse_config(GS_B)), 1).items()}
    toks = random_tokens(GS_B["vocab"], 23, 2)
    whole, streams, _ = pg.forward(GS_B, w, toks)
    assert streams.shape == (6, 23, 50)
    past, parts = None, []
    for a, b in [(0, 9), (9, 11), (11, 23)]:
        logits, _s, past = pg.forward(GS_B, w, toks[a:b], past)
        parts.append(logits)
    assert (torch.cat(parts) - whole).abs().max() < 1e-9


# ====================================================================== kernels on made inputs
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("width", [50, 96, 1024, 4104, 8196])
def test_norm_of_an_output_and_the_next_norm_in_one_launch(dtype, width):
    from helios_b200.csrc import ops
    from helios_b200.parts import LayerNorm, PendingNormed, RMSNorm, settle

    dt = _dt(dtype)
    g = torch.Generator().manual_seed(width)
    res, y = torch.randn(7, width, generator=g) * 3, (torch.randn(7, width, generator=g) * 0.01).to(dt)
    w1, w2 = torch.rand(width, generator=g) + 0.5, torch.rand(width, generator=g) + 0.5
    want = res.double() + pg.rms_norm(y.double(), w1.double(), 1e-4)
    want_out = pg.rms_norm(want, w2.double(), 1e-3)
    tol = 1e-5 if dtype == "float32" else 1e-2
    r = res.cuda()
    out = ops.rmsnorm_add_rmsnorm(r, y.cuda(), w1.cuda(), 1e-4, w2.cuda(), 1e-3)
    assert out.dtype == dt and (r.double().cpu() - want).abs().max() < 1e-5
    assert (out.double().cpu() - want_out).abs().max() < tol * float(want_out.abs().max())
    # wanted rows alone, the stream left as it was
    rows = torch.tensor([5, 0, 5], dtype=torch.int32)
    r = res.cuda()
    out = ops.rmsnorm_add_rmsnorm(r, y.cuda(), w1.cuda(), 1e-4, w2.cuda(), 1e-3, rows.cuda())
    assert torch.equal(r.cpu(), res)
    assert (out.double().cpu() - want_out[rows.long()]).abs().max() < tol * float(want_out.abs().max())
    # a norm of another kind settles what is pending before it
    first = RMSNorm(width, 1e-4)
    first.weight = w1.cuda()
    r = res.cuda()
    settle(r, PendingNormed(y.cuda(), first))
    assert (r.double().cpu() - want).abs().max() < 1e-5
    ln = LayerNorm(width, 1e-5, bias=False)
    ln.weight = w2.cuda()
    r = res.cuda()
    got = ln.add_forward(r, PendingNormed(y.cuda(), first), dt).double().cpu()
    x = want - want.mean(-1, keepdim=True)
    x = x / torch.sqrt((x * x).mean(-1, keepdim=True) + 1e-5) * w2.double()
    assert (got - x).abs().max() < tol * float(x.abs().max())


@pytest.mark.gpu
@pytest.mark.parametrize("n,v", [(1, 7), (3, 448), (2, 5001)])
def test_cap_on_the_logits(n, v):
    from helios_b200.csrc import ops

    x = torch.linspace(-90, 90, n * v).view(n, v)
    got = ops.softcap(x.cuda(), 7.5).double().cpu()
    assert (got - 7.5 * torch.tanh(x.double() / 7.5)).abs().max() < 1e-5


@pytest.mark.gpu
@pytest.mark.parametrize("dtype,T,H,N", [("float32", 5, 3, 6), ("bfloat16", 40, 4, 32), ("bfloat16", 3, 2, 12),
                                         ("bfloat16", 200, 6, 128)])
def test_gate_per_head_on_heads_that_lie_apart(dtype, T, H, N):
    from helios_b200.csrc import ops

    dt = _dt(dtype)
    g = torch.Generator().manual_seed(T)
    x = torch.randn(H, T, N, generator=g).to(dt).cuda().transpose(0, 1)           # head-major storage
    gate = (torch.randn(T, H + 5, generator=g) * 3).to(dt).cuda()
    got = ops.gate_heads(x, gate[:, 3:3 + H], per_head=True).double().cpu().view(T, H, N)
    want = x.double().cpu() * torch.sigmoid(gate[:, 3:3 + H].double().cpu())[:, :, None]
    assert (got - want).abs().max() < (1e-6 if dtype == "float32" else 1e-2) * float(want.abs().max())


def _ctx(parts, slots, tables=None, starts=None, decode=False):
    """A step's description for ops called by hand: ``parts`` tokens per request."""
    from helios_b200.engine.batch import SeqSlice

    starts = starts or [0] * len(parts)
    cu = torch.tensor([0] + list(torch.tensor(parts).cumsum(0)), dtype=torch.int32)
    seq_of = torch.cat([torch.full((n,), i, dtype=torch.int32) for i, n in enumerate(parts)])
    pos = torch.cat([torch.arange(s, s + n, dtype=torch.int32) for s, n in zip(starts, parts)])
    seqs = [SeqSlice(i, slots[i], starts[i], n, int(cu[i])) for i, n in enumerate(parts)]
    ends = [s + n for s, n in zip(starts, parts)]
    return SimpleNamespace(cu_tokens=cu.cuda(), seq_of_token=seq_of.cuda(), positions=pos.cuda(), seqs=seqs,
                           start_pos=torch.tensor(starts, dtype=torch.int32).cuda(),
                           context_len=torch.tensor(ends, dtype=torch.int32).cuda(),
                           slots=torch.tensor(slots, dtype=torch.int32).cuda(), num_seqs=len(parts),
                           num_tokens=int(cu[-1]), max_tokens_per_seq=max(parts), max_context_len=max(ends),
                           decode_only=decode, extras={}, step_tables={}, block_tables=tables or [])


@pytest.mark.gpu
@pytest.mark.parametrize("decays", ["mild", "harsh"])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,N,M,R,tau", [(3, 16, 24, 8, 16.0), (2, 64, 64, 16, 4.0), (4, 7, 33, 5, 1.0),
                                         (2, 130, 65, 3, 2.0), (1, 256, 256, 16, 16.0), (6, 32, 128, 24, 1.0),
                                         (2, 128, 192, 16, 16.0), (3, 100, 48, 1, 0.5)])
def test_recurrence_with_a_decay_per_channel_in_three_steps_from_slots_used_again(dtype, H, N, M, R, tau, decays):
    """Three requests of unequal length in one batch, each cut into three steps at places that are
    and are not borders of a chunk or a sub-chunk; slots zeroed as the cache manager does at
    admission.  Once token by token and once in chunks: both against the plain recurrence in float64,
    the outputs (normed, gated, times a factor) and the states.  ``harsh``: decays down to e^-60 a
    token beside channels that keep everything, whose quotients over a chunk no float32 holds."""
    from helios_b200.csrc import ops

    dt = _dt(dtype)
    g = torch.Generator().manual_seed(H * N + M)
    lengths, cuts, slots = [200, 1, 77], [(64, 129), (1, 1), (3, 21)], [2, 0, 3]
    pad = 5 if dtype == "float32" else 8
    cols = 2 * H * N + 2 * H * M + R
    data = [torch.randn(L, pad + cols, generator=g).to(dt) for L in lengths]
    for d in data:                      # q . k away from 0 on the whole: a norm follows
        d[:, pad:pad + 2 * H * N] += 0.7
    w2 = (torch.randn(H * N, R, generator=g) * R ** -0.5).to(dt)
    bias = torch.randn(H * N, generator=g) + 2.0
    if decays == "harsh":
        bias = torch.where(torch.rand(H * N, generator=g) < 0.5, torch.full((H * N,), 30.0), bias)
        bias = torch.where(torch.rand(H * N, generator=g) < 0.3, torch.full((H * N,), -60.0 * tau), bias)
        w2 = (w2.float() * 4).to(dt)
    weight = torch.rand(M, generator=g) + 0.5
    state0 = torch.randn(5, 4 + H * N * M, generator=g).cuda()
    for s in slots:
        state0[s].zero_()
    q_scale = N ** -0.5

    def run(most):
        kept, ops.LINEAR_ATTENTION_SCAN_TOKENS = ops.LINEAR_ATTENTION_SCAN_TOKENS, most
        state = state0.clone()
        outs = [[] for _ in lengths]
        try:
            for step in range(3):
                cut = [(0,) + c + (L,) for c, L in zip(cuts, lengths)]
                spans = [(c[step], c[step + 1]) for c in cut]
                live = [i for i, (a, b) in enumerate(spans) if b > a]
                rows = torch.cat([data[i][spans[i][0]:spans[i][1]] for i in live]).cuda()
                ctx = _ctx([spans[i][1] - spans[i][0] for i in live], [slots[i] for i in live],
                           starts=[spans[i][0] for i in live])
                wide = torch.full((rows.shape[0], H * M + 16), 7.0, dtype=dt).cuda()
                out = wide[:, 8:8 + H * M]
                offs = (pad, pad + H * N, pad + 2 * H * N, pad + 2 * H * N + H * M, pad + 2 * H * N + 2 * H * M)
                ops.gated_linear_attention(ctx, rows, offs, w2.cuda(), bias.cuda(), tau, state[:, 4:], H, N, M,
                                           weight.cuda(), 1e-4, out, q_scale=q_scale, factor=0.7)
                assert (wide[:, :8] == 7).all() and (wide[:, 8 + H * M:] == 7).all()
                for k, i in enumerate(live):
                    outs[i].append(out[ctx.cu_tokens[k]:ctx.cu_tokens[k + 1]].double().cpu())
        finally:
            ops.LINEAR_ATTENTION_SCAN_TOKENS = kept
        return [torch.cat(o) for o in outs], state.cpu().double()

    mx = {"heads": H, "dim": N, "tau": tau}
    eye = torch.eye(R, dtype=torch.float64)
    W = {"a1": eye, "a2": w2.double(), "a2.b": bias.double()}
    for most in (1 << 30, 0):
        outs, state = run(most)
        for i, d in enumerate(data):
            d = d.double()[:, pad:]
            L = d.shape[0]
            q, k = d[:, :H * N].view(L, H, N), d[:, H * N:2 * H * N].view(L, H, N)
            v = d[:, 2 * H * N:2 * H * N + H * M].view(L, H, M)
            gt = d[:, 2 * H * N + H * M:2 * H * N + 2 * H * M]
            decay = pg.gla_log_decay(d[:, 2 * H * N + 2 * H * M:], W, "", mx)
            o, S = pg.gla_recurrence(q * q_scale, k, v, decay, torch.zeros(H, N, M, dtype=torch.float64))
            want = pg.rms_norm(o, weight.double(), 1e-4).reshape(L, H * M) * gt * torch.sigmoid(gt) * 0.7
            tol = (1e-4 if dtype == "float32" else 2e-2) * max(1.0, float(want.abs().max()))
            assert (outs[i] - want).abs().max() < tol, (most, i, float((outs[i] - want).abs().max()))
            got = state[slots[i], 4:].view(H, N, M)
            assert (got - S).abs().max() < 3e-5 * max(1.0, float(S.abs().max())), (most, i)
        assert torch.equal(state[[1, 4]], state0.cpu().double()[[1, 4]])       # nobody else's slot moved


def _edge_cases(W, n, decode):
    """(query position, key position, visible): the query's own key, the oldest in the window, the one
    before it and the first of all."""
    if decode:
        at = [n - 1, n - 2, 2 * W + 3, W + 15, W, W - 1, W - 2, 16, 15, 1, 0]
    else:
        at = list(range(n - 70, n))
    out = []
    for pos in at:
        if not 0 <= pos < n:
            continue
        picks = [(pos, True), (max(0, pos - W + 1), True), (max(0, pos - W // 2), True)]
        if pos - W >= 0:
            picks += [(pos - W, False), (0, False)]
        out += [(pos, *p) for p in picks] if decode else [(pos, *picks[pos % len(picks)])]
    return out


def _pages_for(keys, values, first_seen, page, dt, g, extra=4):
    """Scrambled pages [pages, heads, page, size] of the rows from ``first_seen`` on, NaN elsewhere, and
    the block table (-1: given back)."""
    n = keys.shape[0]
    n_pages = -(-n // page)
    order = torch.randperm(n_pages + extra, generator=g)[:n_pages]
    kp = torch.full((n_pages + extra, keys.shape[1], page, keys.shape[2]), float("nan"), dtype=dt)
    vp = None if values is None else torch.full((n_pages + extra, values.shape[1], page, values.shape[2]), float("nan"),
                                                dtype=dt)
    for j in range(first_seen // page * page, n):
        kp[order[j // page], :, j % page] = keys[j].to(dt)
        if vp is not None:
            vp[order[j // page], :, j % page] = values[j].to(dt)
    order = order.int()
    order[:first_seen // page] = -1
    return kp.cuda(), None if vp is None else vp.cuda(), order.view(1, -1)


@pytest.mark.gpu
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("dtype,hd,vd,page,W,G", [
    ("float32", 40, 24, 16, 37, 2), ("float32", 16, 16, 8, 1, 1), ("bfloat16", 64, 64, 16, 37, 2),
    ("bfloat16", 128, 128, 16, 44, 4), ("bfloat16", 128, 256, 16, 33, 4), ("bfloat16", 64, 128, 32, 130, 1),
    ("bfloat16", 96, 80, 16, 20, 3), ("bfloat16", 32, 32, 8, 9, 8), ("bfloat16", 128, 64, 16, 1, 5),
    ("bfloat16", 256, 256, 16, 64, 2), ("bfloat16", 192, 128, 16, 50, 16), ("bfloat16", 56, 40, 16, 129, 6),
    ("bfloat16", 20, 36, 16, 30, 2), ("bfloat16", 48, 48, 16, 64, 7)])
def test_window_and_sink_single_out_keys_at_every_edge(dtype, hd, vd, page, W, G, decode):
    """One request of 330 tokens in scrambled pages.  Every query is aligned with ONE key and scaled so
    that this key, if it is visible, takes nearly all the weight but for the sink's share; one that is
    NOT visible must leave no trace.  Pages the window has passed hold NaN.  The sinks run from far
    below the scores to far above them."""
    from helios_b200.csrc import ops

    dt = _dt(dtype)
    g = torch.Generator().manual_seed(7 * hd + vd + W)
    n, nkv = 330, 2
    nh = nkv * G
    unit = torch.randn(n, nkv, hd, generator=g)
    keys = (unit / unit.norm(dim=-1, keepdim=True)).to(dt).float()
    values = torch.randn(n, nkv, vd, generator=g).to(dt).float()
    cases = _edge_cases(W, n, decode)
    q_pos = [c[0] for c in cases]
    first_seen = 0 if decode else max(0, min(q_pos) - W + 1)
    kp, vp, table = _pages_for(keys, values, first_seen, page, dt, g)
    R = len(cases)
    sink = torch.linspace(20.0, 32.0, nh) if nh > 1 else torch.tensor([29.0])
    sink[0] = -1e4
    q = torch.stack([torch.stack([keys[j, h // G] * 60.0 for h in range(nh)]) for _p, j, _v in cases]).to(dt)
    scale = 0.5
    rows = torch.cat([q.view(R, nh * hd), torch.full((R, 8), float("nan"), dtype=dt)], 1).contiguous()   # wider rows
    if decode:
        ctx = _ctx([1] * R, list(range(R)), starts=q_pos, decode=True, tables=[table.repeat(R, 1).contiguous().cuda()])
    else:
        ctx = _ctx([R], [0], starts=[q_pos[0]], tables=[table.cuda()])
    want = torch.stack([pg.window_softmax_attention(q[r:r + 1].double(), keys[:p + 1].double(), values[:p + 1].double(),
                                                    scale, torch.tensor([p]), W, sink.double())[0]
                        for r, p in enumerate(q_pos)])
    for r, (p, j, vis) in enumerate(cases):      # a far sink apart, the case does single out its key
        near = values[j, 0].double()
        assert ((want[r, 0] - near).abs().max() < 0.05 * float(near.abs().max())) == vis
    tol = 2e-5 if dtype == "float32" else 2e-2
    options = ops.AttentionOptions(sink_values=sink.cuda(), value_dim=None if vd == hd else vd)
    for splits in ((None, 1, 2, 5, 8, 11) if decode else (None,)):
        ctx.extras.pop("decode_splits", None)
        if splits:
            ctx.extras["decode_splits"] = splits
        got = ops.attention(ctx, rows.cuda(), kp, vp, ctx.block_tables[0], nh, nkv, hd, page, W, scale, options=options)
        got = got.double().cpu().view(R, nh, vd)
        for r, case in enumerate(cases):
            assert (got[r] - want[r]).abs().max() < tol * max(1.0, float(want[r].abs().max())), (splits, case)


@pytest.mark.gpu
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("dtype,hd,vd,G", [("float32", 10, 14, 3), ("bfloat16", 64, 64, 2), ("bfloat16", 96, 64, 4),
                                           ("bfloat16", 256, 128, 2), ("bfloat16", 40, 72, 1), ("bfloat16", 20, 12, 2)])
def test_query_and_key_norms_cache_write_and_queries_on_anothers_keys(dtype, hd, vd, G, decode):
    """Rows of a fused projection (q | k | v): q and k are normed with their weights, k and v stored,
    and the tokens attend them; then rows of queries ALONE attend the same pages through another
    window and store nothing."""
    from helios_b200.csrc import ops

    dt = _dt(dtype)
    g = torch.Generator().manual_seed(hd + vd)
    nkv, page, eps, scale = 2, 8, 1e-3, 1.2 * hd ** -0.5
    nh = nkv * G
    starts, parts = ([19, 0, 40], [1, 1, 1]) if decode else ([19, 0, 3], [33, 5, 18])
    n = [s + p for s, p in zip(starts, parts)]
    past_k = [torch.randn(s, nkv, hd, generator=g).to(dt) for s in starts]
    past_v = [torch.randn(s, nkv, vd, generator=g).to(dt) for s in starts]
    T = sum(parts)
    width = nh * hd + nkv * (hd + vd)
    pad = -width % 8
    rows = torch.cat([torch.randn(T, width, generator=g), torch.full((T, pad), float("nan"))], 1).to(dt)
    wq, wk = torch.rand(hd, generator=g) * 3 + 0.5, torch.rand(hd, generator=g) + 0.5
    sink = torch.randn(nh, generator=g)
    per = max(-(-x // page) for x in n)
    order = torch.randperm(3 * per + 5, generator=g)[:3 * per].view(3, per)
    kp = torch.full((3 * per + 5, nkv, page, hd), float("nan"), dtype=dt)
    vp = torch.full((3 * per + 5, nkv, page, vd), float("nan"), dtype=dt)
    for i in range(3):
        for j in range(starts[i]):
            kp[order[i, j // page], :, j % page], vp[order[i, j // page], :, j % page] = past_k[i][j], past_v[i][j]
    kp, vp = kp.cuda(), vp.cuda()
    ctx = _ctx(parts, [0, 1, 2], starts=starts, decode=decode, tables=[order.int().cuda()])
    options = ops.AttentionOptions(sink_values=sink.cuda(), value_dim=None if vd == hd else vd)
    got = ops.attention(ctx, rows.clone().cuda(), kp, vp, ctx.block_tables[0], nh, nkv, hd, page, 21, scale,
                        options=options, prepare=(wq.cuda(), wk.cuda(), eps, 0.0, 0, True)).double().cpu()
    lone = torch.randn(T, nh * hd + 8, generator=g).to(dt)
    k_before, v_before = kp.clone(), vp.clone()
    got2 = ops.attention(ctx, lone.clone().cuda(), kp, vp, ctx.block_tables[0], nh, nkv, hd, page, 30, scale,
                         options=options, prepare=(wq.cuda(), None, eps, 0.0, 0, False)).double().cpu()
    same = lambda a, b: torch.equal(torch.nan_to_num(a.float(), nan=-7.0), torch.nan_to_num(b.float(), nan=-7.0))
    assert same(kp, k_before) and same(vp, v_before)
    tol = 3e-5 if dtype == "float32" else 3e-2
    at = 0
    for i, p in enumerate(parts):
        x = rows[at:at + p].double()
        q = pg.rms_norm(x[:, :nh * hd].view(p, nh, hd), wq.double(), eps)
        k = pg.rms_norm(x[:, nh * hd:nh * hd + nkv * hd].reshape(p, nkv, hd), wk.double(), eps)
        v = x[:, nh * hd + nkv * hd:width].reshape(p, nkv, vd)
        for j in range(p):                                   # as stored
            pos = starts[i] + j
            stored = kp[order[i, pos // page], :, pos % page].double().cpu()
            assert (stored - k[j]).abs().max() < tol * float(k.abs().max())
            assert torch.equal(vp[order[i, pos // page], :, pos % page].double().cpu(), v[j])
        kk, vv = torch.cat([past_k[i].double(), k]), torch.cat([past_v[i].double(), v])
        positions = starts[i] + torch.arange(p)
        want = pg.window_softmax_attention(q, kk, vv, scale, positions, 21, sink.double()).reshape(p, -1)
        assert (got[at:at + p] - want).abs().max() < tol * float(want.abs().max()), i
        q = pg.rms_norm(lone[at:at + p, :nh * hd].double().view(p, nh, hd), wq.double(), eps)
        want = pg.window_softmax_attention(q, kk, vv, scale, positions, 30, sink.double()).reshape(p, -1)
        assert (got2[at:at + p] - want).abs().max() < tol * float(want.abs().max()), i
        at += p


@pytest.mark.gpu
@pytest.mark.parametrize("decode", [True, False])
@pytest.mark.parametrize("dtype,H,rank,rot,page,W", [
    ("float32", 3, 20, 6, 16, 37), ("float32", 2, 64, 16, 8, 1), ("bfloat16", 4, 64, 16, 16, 40),
    ("bfloat16", 16, 128, 32, 16, 33), ("bfloat16", 5, 96, 32, 16, 1), ("bfloat16", 40, 32, 16, 32, 130),
    ("bfloat16", 2, 512, 64, 16, 64), ("bfloat16", 3, 20, 6, 8, 31), ("bfloat16", 8, 256, 32, 24, 300)])
def test_latent_window_and_sink_single_out_rows_at_every_edge(dtype, H, rank, rot, page, W, decode):
    """As above, for attention over latent rows: the key is the whole row, the value its first ``rank``
    values; also with the keys of a decode step cut into ranges that are merged."""
    from helios_b200.csrc import ops

    dt = _dt(dtype)
    g = torch.Generator().manual_seed(rank + W)
    n = 1100 if decode and W == 300 else 330
    unit = torch.randn(n, 1, rank + rot, generator=g)
    rows = (unit / unit.norm(dim=-1, keepdim=True)).to(dt).float()
    cases = _edge_cases(W, n, decode)
    q_pos = [c[0] for c in cases]
    first_seen = 0 if decode else max(0, min(q_pos) - W + 1)
    pages, _none, table = _pages_for(rows, None, first_seen, page, dt, g)
    R = len(cases)
    sink = torch.linspace(20.0, 32.0, H)
    sink[0] = -1e4
    q = torch.stack([rows[j].expand(H, -1) * 60.0 for _p, j, _v in cases]).to(dt)
    scale = 0.5
    if decode:
        ctx = _ctx([1] * R, list(range(R)), starts=q_pos, decode=True, tables=[table.repeat(R, 1).contiguous().cuda()])
    else:
        ctx = _ctx([R], [0], starts=[q_pos[0]], tables=[table.cuda()])
    want = torch.stack([pg.window_softmax_attention(q[r:r + 1].double(), rows[:p + 1].double(),
                                                    rows[:p + 1, :, :rank].double(), scale, torch.tensor([p]), W,
                                                    sink.double())[0] for r, p in enumerate(q_pos)])
    for r, (p, j, vis) in enumerate(cases):
        near = rows[j, 0, :rank].double()
        assert ((want[r, 0] - near).abs().max() < 0.05 * float(near.abs().max())) == vis
    qc = q.cuda()
    got = ops.latent_attention(ctx, qc[:, :, :rank], qc[:, :, rank:], pages, ctx.block_tables[0], rank, rot, page, scale,
                               W, sink.cuda()).double().cpu()
    tol = 2e-5 if dtype == "float32" else 2e-2
    for r, case in enumerate(cases):
        assert (got[r] - want[r]).abs().max() < tol * float(want[r].abs().max()), case


@pytest.mark.gpu
@pytest.mark.parametrize("captured", [False, True])
@pytest.mark.parametrize("H,nope,rot,vd,rank,page,W", [
    (4, 32, 16, 32, 64, 16, 40), (3, 128, 64, 128, 512, 16, 130), (5, 40, 24, 16, 96, 8, 17), (2, 64, 32, 64, 128, 32, 1),
    (6, 24, 8, 48, 32, 16, None), (2, 192, 64, 96, 64, 64, 300), (16, 16, 16, 16, 32, 16, 16)])
def test_latent_rows_expanded_to_keys_and_values_per_head(H, nope, rot, vd, rank, page, W, captured):
    """Four requests in one step (a portion deep in a request, a whole prompt, a single token, a portion
    of 16): every query singles out one visible row, or one just outside the window.  Pages the window
    has passed hold NaN and are gone from the tables.  ``captured``: the page count is the bound a
    captured shape takes."""
    from helios_b200.csrc import ops
    from helios_b200.parts.latent_attention import LatentAttention

    g = torch.Generator().manual_seed(H * rank + vd)
    bf = torch.bfloat16
    starts, parts = [333, 0, 210, 61], [70, 145, 1, 16]
    part = LatentAttention(64, H, nope, rot, vd, rank, 0.3, 1e-5, SimpleNamespace(rotary_dim=rot), q_rank=16,
                           pairing="halves", gate="head", window=W, sink=True)
    tensors = {n: torch.randn(s.shape, generator=g).cuda() for n, s in part.weight_specs().items()}
    tensors = {n: (t * rank ** -0.5).to(bf) if part.weight_specs()[n].kind == "matrix" else t for n, t in tensors.items()}
    part.bind(tensors)
    uk, uv = tensors["uk"].double().cpu(), tensors["uv"].double().cpu()
    sink = torch.linspace(-3.0, 25.0, H)
    gate = (torch.randn(sum(parts), H + 3, generator=g) * 2).to(bf)
    tables, q_rows, want, off, pool = [], [], [], 0, []
    most = max(-(-(s + n) // page) for s, n in zip(starts, parts))
    for s, n in zip(starts, parts):
        L = s + n
        rows = torch.randn(L, 1, rank + rot, generator=g).to(bf)
        first = max(0, s - W + 1) if W else 0
        kp, _v, table = _pages_for(rows.float(), None, first, page, bf, g)
        table = torch.where(table >= 0, table + off, table)
        tables.append(torch.cat([table, torch.full((1, most - table.shape[1]), -1, dtype=torch.int32)], 1))
        pool.append(kp)
        off += kp.shape[0]
        x = rows[:, 0].double()
        k = torch.cat([(x[:, :rank] @ uk.T).view(L, H, nope), x[:, None, rank:].expand(L, H, rot)], -1)
        v = (x[:, :rank] @ uv.T).view(L, H, vd)
        targets = [max(0, min(s + i, [s + i, s + i - (W or 200) + 1, s + i - (W or 200), 0, s + i - 3][i % 5])) for i in range(n)]
        q = torch.stack([k[j] / k[j].norm(dim=-1, keepdim=True) * 12.0 for j in targets]).to(bf)
        q_rows.append(q.view(n, -1))
        want.append(pg.window_softmax_attention(q.double(), k, v, 0.3, s + torch.arange(n), W, sink.double()))
    ctx = _ctx(parts, [0, 1, 2, 3], starts=starts, tables=[torch.cat(tables).contiguous().cuda()])
    if captured:
        ctx.extras["tile_provider"] = lambda tile, longest: ops.query_tiles(
            parts, tile, "cuda", starts if longest else None)
    key_dim = nope + rot
    kept, ops.LATENT_EXPAND = ops.LATENT_EXPAND, True
    try:
        n_pages = ops.latent_expand_pages(ctx, H, key_dim, vd, rank, rot, page, W)
    finally:
        ops.LATENT_EXPAND = kept
    exact = sum((s + n - 1) // page - (max(0, s - W + 1) if W else 0) // page + 1 for s, n in zip(starts, parts))
    assert n_pages == exact if not captured else n_pages >= exact
    options = ops.AttentionOptions(sink_values=sink.cuda(), gate=gate.cuda()[:, 2:2 + H])
    wide = torch.cat([torch.cat(q_rows), torch.full((sum(parts), 24), float("nan"), dtype=bf)], 1).cuda()
    got = ops.latent_attention_expanded(ctx, wide[:, :H * key_dim], torch.cat(pool), ctx.block_tables[0],
                                        part.w_expand, n_pages, H, key_dim, vd, page, 0.3, W, options)
    want = torch.cat(want) * torch.sigmoid(gate.double()[:, 2:2 + H])[:, :, None]
    got = got.double().cpu().view(-1, H, vd)
    assert torch.isfinite(got).all()
    err = (got - want).abs().amax(-1) / want.abs().amax()
    assert float(err.max()) < 2.5e-2, (float(err.max()), divmod(int(err.argmax()), H))


# ====================================================================== one key that stands out, in whole models
def _marked_model(kind, W):
    if kind == "attention":
        layers = [(_att(4, 2, 32, 32, 1.0, W), None)]
    elif kind == "other_sizes":
        layers = [(_att(4, 1, 48, 80, 1.0, W), None)]
    elif kind == "borrowed":                              # the reader sees further than the owner of the keys
        layers = [(_att(4, 2, 32, 32, 1.0, 3), None), (_att(4, 2, 32, 32, 1.0, W, kv_from=0), None)]
    else:
        layers = [(_lat(4, 32, 16, 32, 32, 24, 1.0, 1000.0, W), None)]
    return _model(61, 64, 1e-5, 20.0, layers)


def _marked_weights(cfg, weights, A=7, B=9, c0=5, c1=6, mark=3.0, gain=6.0):
    """Token A alone carries a mark in channel c0, which only the key projections read, token B alone
    one in channel c1, which only the query projections read: B's score against A stands far above
    every other, and above the sinks."""
    w = {k: v.clone() for k, v in weights.items()}
    w["embed"] *= 10.0
    w["embed"][:, c0] = w["embed"][:, c1] = 0.0
    w["embed"][A, c0] = w["embed"][B, c1] = mark
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.mix.", layer["mixer"]
        w[f"l{i}.norm1b"][[c0, c1]] = 0.0                 # the marks stay as the embedding left them
        w[f"l{i}.norm1"][[c0, c1]] = 1.0
        d = mx["dim"]
        if layer["type"] == "attention":
            for h in range(mx["heads"]):
                w[p + "q"][h * d + 1, :] = 0.0
                w[p + "q"][h * d + 1, c1] = gain
            w[p + "q.norm"][:] = 3.0
            if "kv_from" not in mx:
                for h in range(mx["kv_heads"]):
                    w[p + "k"][h * d + 1, :] = 0.0
                    w[p + "k"][h * d + 1, c0] = gain
                w[p + "k.norm"][:] = 3.0
        else:
            step = d + mx["rot_dim"]
            w[p + "dq"][0, :] = 0.0
            w[p + "dq"][0, c1] = gain                     # the query latent's value 0 carries B's mark ...
            w[p + "uq"][:, 0] = 0.0
            w[p + "uk"][:, 0] = 0.0
            for h in range(mx["heads"]):                  # ... into unrotated value 0 of every head's query
                w[p + "uq"][h * step, :] = 0.0
                w[p + "uq"][h * step, 0] = gain
                w[p + "uk"][h * d, :] = 0.0               # and the latent's value 0 into that value of the key
                w[p + "uk"][h * d, 0] = gain
            w[p + "dkv"][0, :] = 0.0
            w[p + "dkv"][0, c0] = gain                    # the latent's value 0 carries A's mark
    return w


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", ["attention", "other_sizes", "borrowed", "latent"])
def test_one_key_just_inside_and_just_outside_the_window(kind, dtype, tmp_path):
    """The marked key as the window's oldest, one before it, at a page's last place and the next
    page's first, far outside; the marked query in a prompt, in a later portion, and decoded alone."""
    from conftest import assert_logits_close
    from safetensors.torch import save_file
    from helios_b200.engine.batch import StepEntry
    from helios_b200.weights import write_model_folder

    W, n = 90, 301
    cfg = _marked_model(kind, W)
    folder = write_model_folder(tmp_path / kind, cfg, 11)
    _c, weights = read_folder(folder)
    weights = _marked_weights(cfg, weights)
    save_file(weights, str(folder / "model.safetensors"))
    w = _weights(weights, dtype)
    A, B = 7, 9
    filler = [t for t in random_tokens(cfg["vocab"], 2 * n, 5) if t not in (A, B)][:n]
    core = _core(folder, dtype, 1024)
    last = n - 1
    plain = {}
    for case, where in enumerate([last - W + 1, last - W, 0, 223, 224, last - 1, last - W + 2, last - W - 1, 250]):
        toks = list(filler)
        toks[where], toks[last] = A, B
        want = pg.forward(cfg, w, toks)[0]
        toks[where] = filler[where]
        moved = (want[last] - pg.forward(cfg, w, toks)[0][last]).abs().max() / want[last].abs().max()
        assert (float(moved) > 0.05) == (last - where < W), (where, float(moved))     # the key shows where it is seen
        toks[where] = A
        for k, cuts in enumerate([[n], [last, 1], [where + 1, last - where - 1, 1], [16, 17, n - 33 - 40] + [1] * 40]):
            rid, at = f"{kind}{case}.{k}", 0
            for c in [c for c in cuts if c > 0]:
                got = core.step([StepEntry(rid, toks[at:at + c], [c - 1])])
                at += c
            core.end(rid)
            assert_logits_close(got, want[last:], dtype, f"{kind}: key at {where}, cuts {cuts[:4]}")


# ====================================================================== whole models
@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(GS_ALONE) + list(GS_CONFIGS))
def test_whole_prompts_and_the_stream_after_every_layer(gs_folders, name, dtype):
    """Logits at every position of whole prompts (the first tokens of a sequence among them), and
    the residual stream after every layer."""
    from helios_b200.engine.batch import StepEntry

    cfg, weights = read_folder(gs_folders[name])
    reqs = _requests(cfg, [1, 2, 3, 41, 200], 100)
    plain = _plain(cfg, weights, dtype, reqs)
    tb = tu.TraceBuilder()
    for rid, toks in reqs.items():
        tu.whole(tb, rid, toks)
    core = _core(gs_folders[name], dtype, tb.live_tokens_peak)
    _check(tb, tu.run_in_process(core, tb), plain, dtype, f"{name} whole")
    _, want_layers, _ = pg.forward(cfg, _weights(weights, dtype), reqs["q3"])
    seen = []

    def recording(inner):
        def forward(*args):
            residual, pending = inner(*args)
            y, norm = pending.y.double().cpu(), pending.norm
            seen.append(residual.double().cpu() + pg.rms_norm(y, norm.weight.double().cpu(), norm.eps))
            return residual, pending
        return forward

    for blk in core.model.plan.layers:
        blk.forward = recording(blk.forward)
    core.step([StepEntry("layers", reqs["q3"], [0])])
    assert len(seen) == want_layers.shape[0]
    for i, (got, want) in enumerate(zip(seen, want_layers)):
        tol = 2e-5 * max(1.0, float(want.abs().max())) if dtype == "float32" else 3e-2 * float(want.abs().max())
        assert (got - want).abs().max() < tol, f"{name}: residual after layer {i}"


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(GS_CONFIGS))
def test_prefill_then_long_decoding_token_by_token(gs_folders, name, dtype):
    """Most of the prompt in one step, then 110 single tokens (captured decode steps) that pass page
    borders and whole windows, up to position 300."""
    cfg, weights = read_folder(gs_folders[name])
    reqs = _requests(cfg, [115, 171, 300], 200)
    plain = _plain(cfg, weights, dtype, reqs)
    tb = tu.TraceBuilder()
    for rid, toks in reqs.items():
        tu.prefill_then_decode(tb, rid, toks, n_decode=110)
    core = _core(gs_folders[name], dtype, tb.live_tokens_peak)
    _check(tb, tu.run_in_process(core, tb), plain, dtype, f"{name} decode")


@pytest.mark.gpu
@pytest.mark.parametrize("page", [16, 4])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(GS_CONFIGS))
def test_portions_of_changing_size_down_to_one_token(gs_folders, name, dtype, page):
    cfg, weights = read_folder(gs_folders[name])
    reqs = _requests(cfg, [64, 197, 50, 33], 300)
    plain = _plain(cfg, weights, dtype, reqs)
    tb = tu.TraceBuilder()
    sizes = [[7], [2, 31, 3, 16, 2, 17, 40], [1, 2, 1, 1, 3, 13, 2, 1, 5], [16, 1, 15, 1]]
    for (rid, toks), sz in zip(reqs.items(), sizes):
        tu.portions(tb, rid, toks, sz)
    core = _core(gs_folders[name], dtype, tb.live_tokens_peak, page_size=page)
    _check(tb, tu.run_in_process(core, tb), plain, dtype, f"{name} portions")


@pytest.mark.gpu
@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", list(GS_CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(gs_folders, name, dtype, graphs):
    """Nine unequal requests through three slots: portions of some beside single tokens of others;
    every finished request's pages and slot go to the next."""
    cfg, weights = read_folder(gs_folders[name])
    reqs = _requests(cfg, [40, 23, 177, 18, 52, 31, 66, 20, 45], 400)
    plain = _plain(cfg, weights, dtype, reqs)
    tb = tu.TraceBuilder()
    tu.mixed(tb, reqs, seed=7, max_live=3, decode_tail=10)
    core = _core(gs_folders[name], dtype, tb.live_tokens_peak, max_slots=3, graphs=graphs)
    _check(tb, tu.run_in_process(core, tb), plain, dtype, f"{name} mixed")
    assert core.cache.num_free_slots == 3 and all(p.num_used == 0 for p in core.cache.pools)


@pytest.mark.gpu
@pytest.mark.parametrize("graphs", [True, False])
@pytest.mark.parametrize("name", ["latent_only", "gs_a", "gs_c"])
def test_models_whose_portions_expand_their_latent_rows(gs_folders, name, graphs, monkeypatch):
    """Portions of 16 tokens and more by way of keys and values per head, beside decoded tokens and
    shorter portions that attend the rows themselves."""
    from helios_b200.csrc import ops

    made = []
    monkeypatch.setattr(ops, "LATENT_EXPAND", True)
    inner = ops.latent_attention_expanded
    monkeypatch.setattr(ops, "latent_attention_expanded", lambda *a, **kw: made.append(1) or inner(*a, **kw))
    cfg, weights = read_folder(gs_folders[name])
    reqs = _requests(cfg, [140, 23, 277, 18, 52, 131], 700)
    plain = _plain(cfg, weights, "bfloat16", reqs)
    tb = tu.TraceBuilder()
    tu.mixed(tb, reqs, seed=5, max_live=3, decode_tail=10, portion_choices=(2, 16, 40, 70))
    core = _core(gs_folders[name], "bfloat16", tb.live_tokens_peak, max_slots=3, graphs=graphs)
    _check(tb, tu.run_in_process(core, tb), plain, "bfloat16", f"{name} expanded")
    assert made


@pytest.mark.gpu
@pytest.mark.parametrize("name", ["gs_a", "gs_b", "gs_c"])
def test_a_batch_gives_each_request_what_it_gets_alone(gs_folders, name):
    """float32: the same rows alone or beside others, in one step or in portions, whatever the slots
    and pages, up to rounding (a portion's borders are borders of the recurrence's chunks)."""
    from helios_b200.engine.batch import StepEntry

    cfg, _w = read_folder(gs_folders[name])
    reqs = _requests(cfg, [37, 5, 160], 500)
    core = _core(gs_folders[name], "float32", 512, max_slots=4)
    alone = {}
    for rid, toks in reqs.items():
        alone[rid] = core.step([StepEntry(rid, toks, range(len(toks)))]).clone()
        core.end(rid)
    core.step([StepEntry("other", random_tokens(cfg["vocab"], 21, 1), [0])])      # shifts slots and pages
    got = core.step([StepEntry(rid, toks, range(len(toks))) for rid, toks in reqs.items()])
    off = 0
    for rid, toks in reqs.items():
        assert (got[off:off + len(toks)] - alone[rid]).abs().max() < 6e-6, rid
        off += len(toks)
    for rid in reqs:
        core.end(rid)
    toks = reqs["q2"]
    cuts = [0, 2, 31, 33, 97, 160]
    parts = [core.step([StepEntry("cut", toks[a:b], range(b - a))]) for a, b in zip(cuts, cuts[1:])]
    assert (torch.cat(parts) - alone["q2"]).abs().max() < 6e-6


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
def test_through_trace_run(gs_folders, dtype, tmp_path):
    cfg, weights = read_folder(gs_folders["gs_b"])
    reqs = _requests(cfg, [30, 47, 22, 39, 128], 600)
    plain = _plain(cfg, weights, dtype, reqs)
    tb = tu.TraceBuilder()
    tu.mixed(tb, reqs, seed=3, max_live=4, decode_tail=8)
    got = tu.run_trace_run(gs_folders["gs_b"], dtype, tb, tmp_path / "out", tb.live_tokens_peak, cfg["vocab"])
    _check(tb, got, plain, dtype, "gs_b trace_run")


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["gs_a", "gs_b"])
def test_greedy_generation_through_the_scheduler(gs_folders, name, dtype):
    from helios_b200 import LLM, SamplingParams

    cfg, weights = read_folder(gs_folders[name])
    w = _weights(weights, dtype)
    prompts = [random_tokens(cfg["vocab"], n, 40 + n) for n in (1, 5, 17, 33, 9, 60)]
    llm = LLM(str(gs_folders[name]), dtype=dtype, kv_cache_bytes=1 << 22, max_num_batched_tokens=24,
              max_num_seqs=4, max_model_len=256)
    outs = llm.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(max_tokens=12))
    for prompt, out in zip(prompts, outs):
        assert out.completion_tokens == 12
        toks = list(prompt) + list(out.token_ids)
        logits = pg.forward(cfg, w, toks)[0][len(prompt) - 1:-1]        # one pass: causal
        for i, t in enumerate(out.token_ids):
            best = int(torch.argmax(logits[i]))
            if t != best:
                assert dtype == "bfloat16", f"token {t} instead of {best} at {i}"
                assert float(logits[i, best] - logits[i, t]) <= 0.03 * float(logits[i].abs().max())


@pytest.mark.gpu
def test_a_pool_too_small_for_all_requests_gives_pages_from_one_to_the_next(gs_folders):
    """Generation through a pool that holds about two of six requests: nobody's tokens change."""
    from helios_b200 import LLM, SamplingParams

    cfg, _w = read_folder(gs_folders["gs_b"])
    prompts = [random_tokens(cfg["vocab"], n, 70 + n) for n in (50, 31, 64, 12, 45, 28)]
    llm = LLM(str(gs_folders["gs_b"]), dtype="float32", kv_cache_bytes=1 << 24, max_num_seqs=6, max_model_len=128)
    want = [o.token_ids for o in llm.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(max_tokens=20))]
    tight = LLM(str(gs_folders["gs_b"]), dtype="float32", num_blocks=22, block_size=8, max_num_seqs=6,
                max_num_batched_tokens=32, max_model_len=128, watermark=0.0)
    got = [o.token_ids for o in tight.generate(prompt_token_ids=prompts, sampling_params=SamplingParams(max_tokens=20))]
    assert got == want


# ====================================================================== configurations drawn at random
def draw_config(seed):
    """Sizes, head counts, layer order, windows, borrowers and constants at random."""
    rng = random.Random(seed)
    dims = (8, 12, 16, 24, 32, 40, 48, 64, 80, 96, 128, 160, 192)
    window = lambda: rng.choice([1, 2, 7, 16, 17, 33, 64, 100, 130, 200])
    layers = []
    for i in range(rng.randint(2, 5)):
        own = [j for j, (l, _ff) in enumerate(layers) if l["type"] == "attention" and "kv_from" not in l["mixer"]]
        kind = rng.choice(["attention", "gla", "latent"])
        if own and rng.random() < 0.4:
            src = rng.choice(own)
            mx = layers[src][0]["mixer"]
            layer = _att(mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["scale"], window(), kv_from=src)
        elif kind == "attention":
            d, kv = rng.choice(dims), rng.choice([1, 2, 3])
            layer = _att(kv * rng.choice([1, 2, 4, 5, 8]), kv, d, rng.choice(dims),
                         round(rng.uniform(0.5, 2.0) * d ** -0.5, 4), window())
        elif kind == "gla":
            layer = _gla(rng.randint(1, 6), rng.choice(dims), rng.choice(dims), rng.choice([1.0, 2.0, 8.0, 16.0]),
                         rng.choice([1, 4, 6, 16, 32]))
        else:
            d, rot = rng.choice(dims[:10]), rng.choice([2, 8, 16, 32, 64])
            layer = _lat(rng.randint(1, 9), d, rot, rng.choice(dims[:10]), rng.choice([12, 32, 64, 96, 128, 256]),
                         rng.choice([5, 24, 64, 128]), round(rng.uniform(0.5, 2.0) * (d + rot) ** -0.5, 4),
                         rng.choice([50.0, 5e3, 5e5]), window())
        layers.append((layer, rng.choice([None, 24, 64, 136])))
    return _model(rng.randint(40, 700), 8 * rng.randint(3, 40), rng.choice([1e-5, 1e-6, 3e-6]),
                  rng.choice([None, 1.5, 5.0, 30.0]), layers), rng


@pytest.mark.gpu
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("seed", range(8))
def test_a_random_configuration_matches_the_plain_implementation(tmp_path, seed, dtype):
    compare_random(tmp_path, seed, dtype)


def compare_random(tmp_path, seed, dtype, lengths=(70, 23, 250)):
    from safetensors.torch import save_file
    from helios_b200.weights import write_model_folder

    cfg, rng = draw_config(seed)
    folder = write_model_folder(tmp_path / "m", cfg, seed)
    _cfg, weights = read_folder(folder)
    weights = _lively(cfg, weights)
    save_file(weights, str(folder / "model.safetensors"))
    _write_lean(folder, cfg)
    reqs = _requests(cfg, lengths, 1000 + seed)
    plain = _plain(cfg, weights, dtype, reqs)
    tb = tu.TraceBuilder()
    tu.mixed(tb, reqs, seed=seed, max_live=2, decode_tail=12, portion_choices=(2, 3, 9, 34, 70))
    core = _core(folder, dtype, tb.live_tokens_peak, page_size=rng.choice([16, 16, 8, 32]), max_slots=2)
    _check(tb, tu.run_in_process(core, tb), plain, dtype, f"seed {seed}", most=0.06, outliers=0.05)
