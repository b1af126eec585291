"""A plain, slow float64 implementation of the Mozepel design, written from its equations: one
function per mechanism, whole sequences only, no cache, no state between calls, no code
shared with the package.  ``tensors`` maps checkpoint names to float64 tensors; ``cfg`` is the
dictionary of ``config.json``.

Notation: T tokens, positions 0..T-1, h the input of a sublayer ([T, width]).
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def silu(z):
    return z * torch.sigmoid(z)


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms_unit(x, eps) * w


def frequencies(rot):
    """One frequency per rotated pair: base^(-2i/dims), stretched by wavelength where the
    file asks for it (long waves divided by ``factor``, short ones kept, a linear blend of the
    two in between)."""
    half = rot["dims"] // 2
    out = []
    for i in range(half):
        f = float(rot["base"]) ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc:
            wave = 2.0 * math.pi / f
            if wave < sc["original"] / sc["high"]:
                pass
            elif wave > sc["original"] / sc["low"]:
                f = f / sc["factor"]
            else:
                s = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return torch.tensor(out, dtype=F64)


def rotate_half(x, positions, rot):
    """x [T, heads, dim]: the first rot.dims values of every head rotated, value i paired with
    value i + dims/2."""
    half = rot["dims"] // 2
    ang = positions.to(F64)[:, None] * frequencies(rot)[None, :]
    c, s = torch.cos(ang)[:, None, :], torch.sin(ang)[:, None, :]
    u, v = x[..., :half], x[..., half:2 * half]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., 2 * half:]], dim=-1)


def causal_conv(x, w):
    """x [T, C], w [C, taps] (last column: the current token), zeros before the start."""
    T, C = x.shape
    taps = w.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, C, dtype=x.dtype), x], dim=0)
    y = torch.zeros(T, C, dtype=x.dtype)
    for j in range(taps):
        y = y + padded[j:j + T] * w[:, j]
    return y


def fixed_decay(q, k, v, decay):
    """q, k [T, H, n], v [T, H, m]: token by token and head by head S <- decay S + k v^T from
    S = 0, o = S^T q; returns o [T, H, m]."""
    T, H, n = q.shape
    lam = torch.as_tensor(decay, dtype=F64)[:, None, None]
    S = torch.zeros(H, n, v.shape[-1], dtype=F64)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = lam * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def retention_mixer(h, t, p, mx, eps):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    pos = torch.arange(T)
    q = rotate_half((h @ t[p + "q"].T).view(T, H, d), pos, mx["rot"])
    k = rotate_half((h @ t[p + "k"].T).view(T, H, d), pos, mx["rot"]) * d ** -0.5
    v = (h @ t[p + "v"].T).view(T, H, dv)
    o = rms_unit(fixed_decay(q, k, v, mx["decay"]), eps).reshape(T, H * dv)
    return (o * silu(h @ t[p + "g"].T)) @ t[p + "o"].T


def lightning_mixer(h, t, p, mx, eps):
    T = h.shape[0]
    H, d, dv = mx["heads"], mx["dim"], mx["vdim"]
    q = silu(h @ t[p + "q"].T).view(T, H, d)
    k = silu(h @ t[p + "k"].T).view(T, H, d)
    v = silu(h @ t[p + "v"].T).view(T, H, dv)
    o = rms_norm(fixed_decay(q, k, v, mx["decay"]).reshape(T, H * dv), t[p + "norm"], eps)
    return (o * torch.sigmoid(h @ t[p + "g"].T)) @ t[p + "o"].T


def pooled_window_weights(scores, pooled_scores, size, pool):
    """Softmax over the last ``size`` tokens and, beside them, over the whole blocks of ``pool``
    tokens that lie before the window: scores [T, T] and pooled_scores [T, blocks] ->
    weights of the same shapes."""
    T = scores.shape[0]
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    see = (j <= i) & (i - j < size)
    last = torch.arange(pooled_scores.shape[1])[None, :] * pool + pool - 1
    see_block = last <= i - size
    s = torch.cat([scores.masked_fill(~see, -math.inf), pooled_scores.masked_fill(~see_block, -math.inf)], dim=1)
    w = torch.softmax(s, dim=1)
    return w[:, :T], w[:, T:]


def window_mixer(h, t, p, mx, eps):
    T = h.shape[0]
    H, G, d, dv = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    pos = torch.arange(T)

    def project(name, heads, width):
        u = h @ t[p + name].T
        if p + name + ".conv" in t:
            u = causal_conv(u, t[p + name + ".conv"])
        return u.view(T, heads, width)

    q = rotate_half(rms_norm(project("q", H, d), t[p + "q.norm"], eps), pos, mx["rot"])
    k = rotate_half(rms_norm(project("k", G, d), t[p + "k.norm"], eps), pos, mx["rot"])
    v = project("v", G, dv)
    P = mx["mask"].get("pool") or T + 1          # without blocks: one that is never whole
    nb = T // P
    kp = k[:nb * P].view(nb, P, G, d).mean(1)
    vp = v[:nb * P].view(nb, P, G, dv).mean(1)
    out = torch.zeros(T, H, dv, dtype=F64)
    for hh in range(H):
        g = hh // (H // G)
        w, wp = pooled_window_weights(q[:, hh] @ k[:, g].T * mx["scale"], q[:, hh] @ kp[:, g].T * mx["scale"],
                                      mx["mask"]["size"], P)
        out[:, hh] = w @ v[:, g] + wp @ vp[:, g]
    return out.reshape(T, H * dv) @ t[p + "o"].T


def parallel_mixer(h, t, p, mx, eps):
    return (mx["left_scale"] * window_mixer(h, t, p + "left.", mx["left"], eps)
            + mx["right_scale"] * lightning_mixer(h, t, p + "right.", mx["right"], eps))


MIXERS = {"retention": retention_mixer, "parallel": parallel_mixer}


def dense_ff(h, t, p):
    return (silu(h @ t[p + "gate"].T) * (h @ t[p + "up"].T)) @ t[p + "down"].T


def norm_after_sum(x, y, w, alpha, eps):
    return rms_norm(alpha * x + y, w, eps)


def model(cfg, tensors, tokens):
    """(logits [T, vocab], the stream after every layer run [runs, T, width])."""
    t = tensors
    eps, alpha = cfg["norm"]["eps"], cfg["postln_alpha"]
    x = t["embed"][torch.as_tensor(list(tokens))]
    stream = []
    for i, layer in enumerate(cfg["layers"]):
        j = i if layer.get("weights_of") is None else layer["weights_of"]
        p = f"l{j}."
        x = norm_after_sum(x, MIXERS[layer["type"]](x, t, p + "mix.", layer["mixer"], eps), t[p + "norm1"], alpha, eps)
        if layer.get("mlp"):
            x = norm_after_sum(x, dense_ff(x, t, p + "mlp."), t[p + "norm2"], alpha, eps)
        stream.append(x)
    return rms_norm(x, t["final.norm"], eps) @ t["head"].T, torch.stack(stream)
