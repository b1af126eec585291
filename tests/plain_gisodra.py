"""Plain, slow float64 implementation of the Gisodra design, one function per mechanism, written
from the design's equations with torch on the CPU.  It shares no code with the package: it reads
``config.json`` as a dictionary and the checkpoint by tensor name.

Notation: x [T, width] is the residual stream.  A layer norms before AND after each sublayer:
x <- x + norm1b(mixer(norm1(x))), x <- x + norm2b(ff(norm2(x))); the feed-forward may be absent.
``W`` maps a tensor's name to a float64 tensor, ``p`` is a prefix such as ``l3.mix.``.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms_norm(x, weight, eps):
    """x / sqrt(mean(x^2) + eps) * weight over the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def rotate_halves(x, positions, dims, base):
    """The first ``dims`` values of the last dimension, value i paired with value i + dims / 2:
    (u, v) -> (u cos a - v sin a, v cos a + u sin a), a = position * base^(-2 i / dims).
    x [T, ..., d]."""
    half = dims // 2
    a = positions.to(F64)[:, None] * base ** (-2.0 * torch.arange(half, dtype=F64) / dims)[None, :]
    c, s = torch.cos(a), torch.sin(a)
    while c.dim() < x.dim():
        c, s = c.unsqueeze(1), s.unsqueeze(1)
    out = x.clone()
    u, v = x[..., :half], x[..., half:dims]
    out[..., :half] = u * c - v * s
    out[..., half:dims] = v * c + u * s
    return out


def window_softmax_attention(q, k, v, scale, positions, window, sink):
    """q [T, H, d], k [S, G, d], v [S, G, dv] with key j at position j; the query of row t at
    i = positions[t] sees the keys 0 <= i - j < window (None: every j <= i).  The softmax's
    denominator has one more term, exp(sink[h]).  Head h reads key/value head h // (H / G)."""
    T, H, _ = q.shape
    S, G, _ = k.shape
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    dist = positions[:, None] - torch.arange(S)[None, :]
    hidden = (dist < 0) | ((dist >= window) if window is not None else torch.zeros_like(dist, dtype=torch.bool))
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].T) * scale).masked_fill(hidden, -math.inf)
        top = torch.maximum(s.max(-1).values, sink[h])[:, None]
        e = torch.exp(s - top)
        out[:, h] = (e / (e.sum(-1, keepdim=True) + torch.exp(sink[h] - top))) @ v[:, g]
    return out


def _window(mx):
    mask = mx.get("mask")
    return mask["size"] if mask else None


# ---------------------------------------------------------------------- attention
def attention_rows(h, W, p, mx, eps):
    """What an attention layer keeps per token: k [T, G, d] normed per head, v [T, G, dv]."""
    G, d, dv = mx["kv_heads"], mx["dim"], mx["vdim"]
    k = (h @ W[p + "k"].T + W[p + "k.b"]).view(-1, G, d)
    v = (h @ W[p + "v"].T + W[p + "v.b"]).view(-1, G, dv)
    return rms_norm(k, W[p + "k.norm"], eps), v


def attention_mixer(h, W, p, mx, eps, past=None, borrowed=None):
    """No rotation.  ``borrowed`` = (k, v) of ALL tokens so far as another layer keeps them; else
    ``past`` = those of the tokens before h's.  Returns (out, (k, v))."""
    T = h.shape[0]
    if borrowed is not None:
        k, v = borrowed
    else:
        k, v = attention_rows(h, W, p, mx, eps)
        if past is not None:
            k, v = torch.cat([past[0], k]), torch.cat([past[1], v])
    positions = k.shape[0] - T + torch.arange(T)
    q = rms_norm((h @ W[p + "q"].T + W[p + "q.b"]).view(T, mx["heads"], mx["dim"]), W[p + "q.norm"], eps)
    o = window_softmax_attention(q, k, v, mx["scale"], positions, _window(mx), W[p + "sink"])
    return o.reshape(T, -1) @ W[p + "o"].T, (k, v)


# ---------------------------------------------------------------------- gated linear attention
def gla_log_decay(h, W, p, mx):
    """ln of the decay per token, head and key channel: logsigmoid(W_a2 (W_a1 h) + b) / tau."""
    z = (h @ W[p + "a1"].T) @ W[p + "a2"].T + W[p + "a2.b"]
    return -torch.nn.functional.softplus(-z, threshold=1e9).view(-1, mx["heads"], mx["dim"]) / mx["tau"]


def gla_recurrence(q, k, v, log_decay, state):
    """Token by token, per head: S <- diag(exp(log_decay)) S + k v^T, o = S^T q.  q, k, log_decay
    [T, H, d], v [T, H, dv], state [H, d, dv].  Returns (o [T, H, dv], state)."""
    S = state.clone()
    out = []
    for t in range(q.shape[0]):
        S = torch.exp(log_decay[t])[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdm,hd->hm", S, q[t]))
    return torch.stack(out), S


def gla_mixer(h, W, p, mx, eps, past=None):
    T, H, d, dv = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, d) * d ** -0.5
    k = (h @ W[p + "k"].T).view(T, H, d)
    v = (h @ W[p + "v"].T).view(T, H, dv)
    state = torch.zeros(H, d, dv, dtype=F64) if past is None else past
    o, state = gla_recurrence(q, k, v, gla_log_decay(h, W, p, mx), state)
    o = rms_norm(o, W[p + "norm"], eps).reshape(T, -1)
    g = h @ W[p + "g"].T
    return (o * g * torch.sigmoid(g)) @ W[p + "o"].T, state


# ---------------------------------------------------------------------- latent attention
def latent_rows(h, W, p, mx, eps, positions):
    """What a latent layer keeps per token: the normed latent c [T, rank] and the shared key
    part [T, rot_dim], rotated."""
    r = mx["kv_rank"]
    both = h @ W[p + "dkv"].T
    c = rms_norm(both[:, :r], W[p + "dkv.norm"], eps)
    return c, rotate_halves(both[:, r:], positions, mx["rot"]["dims"], mx["rot"]["base"])


def latent_mixer(h, W, p, mx, eps, past=None):
    """Queries through a normed latent of their own; per head the key is [W_uk c | shared rotated
    part] and the value W_uv c; head h's output is multiplied by sigmoid(W_g h)_h."""
    T = h.shape[0]
    H, dn, dr, dv = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    n0 = 0 if past is None else past[0].shape[0]
    positions = n0 + torch.arange(T)
    cq = rms_norm(h @ W[p + "dq"].T, W[p + "dq.norm"], eps)
    q = (cq @ W[p + "uq"].T).view(T, H, dn + dr)
    q = torch.cat([q[..., :dn], rotate_halves(q[..., dn:], positions, mx["rot"]["dims"], mx["rot"]["base"])], dim=-1)
    c, kr = latent_rows(h, W, p, mx, eps, positions)
    if past is not None:
        c, kr = torch.cat([past[0], c]), torch.cat([past[1], kr])
    S = c.shape[0]
    k = torch.cat([(c @ W[p + "uk"].T).view(S, H, dn), kr[:, None, :].expand(S, H, dr)], dim=-1)
    v = (c @ W[p + "uv"].T).view(S, H, dv)
    o = window_softmax_attention(q, k, v, mx["scale"], positions, _window(mx), W[p + "sink"])
    o = o * torch.sigmoid(h @ W[p + "g"].T)[:, :, None]
    return o.reshape(T, -1) @ W[p + "o"].T, (c, kr)


# ---------------------------------------------------------------------- feed-forward, model
def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def dense_ff(h, W, p):
    return (gelu_tanh(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, W, tokens, past=None):
    """tokens: list of ids that follow what ``past`` holds (None: the start of a request).
    Returns (logits [T, vocab], streams [layers, T, width], past)."""
    W = {k: v.to(F64) for k, v in W.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.tensor(tokens, dtype=torch.long)]
    past = past or {}
    kept, streams = {}, []
    for i, layer in enumerate(cfg["layers"]):
        p, mx = f"l{i}.mix.", layer["mixer"]
        h = rms_norm(x, W[f"l{i}.norm1"], eps)
        if layer["type"] == "attention" and mx.get("kv_from") is not None:
            m, _ = attention_mixer(h, W, p, mx, eps, borrowed=kept[mx["kv_from"]])
        elif layer["type"] == "attention":
            m, kept[i] = attention_mixer(h, W, p, mx, eps, past.get(i))
        elif layer["type"] == "latent_attention":
            m, kept[i] = latent_mixer(h, W, p, mx, eps, past.get(i))
        elif layer["type"] == "gla":
            m, kept[i] = gla_mixer(h, W, p, mx, eps, past.get(i))
        else:
            raise ValueError(layer["type"])
        x = x + rms_norm(m, W[f"l{i}.norm1b"], eps)
        if layer.get("mlp") is not None:
            f = dense_ff(rms_norm(x, W[f"l{i}.norm2"], eps), W, f"l{i}.mlp.")
            x = x + rms_norm(f, W[f"l{i}.norm2b"], eps)
        streams.append(x)
    logits = rms_norm(x, W["final.norm"], eps) @ W["embed"].T
    cap = cfg.get("logit_softcap")
    if cap:
        logits = cap * torch.tanh(logits / cap)
    return logits, torch.stack(streams), kept
