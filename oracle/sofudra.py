"""Plain, slow restatement of the Sofudra decoders (numpy), one function per mechanism.

Test infrastructure, like oracle/hybrid.py, whose elementary functions it uses: everything is written from the equations
over whole sequences, without caches, chunks or code of the product.

A model is a dict {"config": a checkpoint's config.json as a dict, "tensors": {name: array}}. `rnd` rounds the operands of
matrix products (identity by default).
"""
from __future__ import annotations

import math

import numpy as np

from .hybrid import exact, rms_norm, sigmoid, silu


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def softcap(z, cap):
    return cap * np.tanh(z / cap)


def rotary_frequencies(rot):
    """(frequencies [dims / 2], factor of cos and sin) of a rotation, with YaRN scaling where it has one."""
    dims, base = rot["dims"], rot["base"]
    i = np.arange(dims // 2, dtype=np.float64)
    f = float(base) ** (-2.0 * i / dims)
    sc = rot.get("scaling")
    if not sc:
        return f, 1.0

    def turns_to_dim(t):
        return dims * math.log(sc["original"] / (2.0 * math.pi * t)) / (2.0 * math.log(base))
    lo = max(math.floor(turns_to_dim(sc["fast"])), 0)
    hi = min(math.ceil(turns_to_dim(sc["slow"])), dims - 1)
    ramp = np.clip((i - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / sc["factor"] * ramp + f * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate(x, pos, rot):
    """Entries i and i + dims / 2 of the last axis turn by pos * f_i. x [T, heads, n], pos [T]."""
    f, mul = rotary_frequencies(rot)
    half = rot["dims"] // 2
    a = (pos[:, None] * f)[:, None, :]
    c, s = (np.cos(a) * mul).astype(x.dtype), (np.sin(a) * mul).astype(x.dtype)
    u, v = x[..., :half], x[..., half:2 * half]
    return np.concatenate([u * c - v * s, v * c + u * s, x[..., 2 * half:]], axis=-1)


def attend(q, k, v, scale, window=0, cap=0.0, sink=None, rnd=exact):
    """Causal attention of one head: q, k [T, d], v [T, n]. A sink is one more term of the denominator."""
    T = q.shape[0]
    s = (q @ k.T) * scale
    if cap:
        s = softcap(s, cap)
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    ok = (j <= i) & (i - j < window) if window else (j <= i)
    s = np.where(ok, s, -np.inf)
    m = s.max(-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    p = np.exp(s - m)
    den = p.sum(-1, keepdims=True)
    if sink is not None:
        den = den + np.exp(sink - m)
    return rnd(p / den) @ v


def attention_mixer(h, mx, W, has, eps, rnd=exact):
    """Softmax attention with grouped heads; what a layer has beyond that is read off its tensors and constants."""
    h = rnd(h)
    T, H, G, D, V = h.shape[0], mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]

    def proj(n, heads, size):
        y = h @ W(n).T
        if has(n + ".b"):
            y = y + W(n + ".b")
        return y.reshape(T, heads, size)
    q, k, v = proj("q", H, D), proj("k", G, D), proj("v", G, V)
    if has("q.norm"):
        q, k = rms_norm(q, W("q.norm"), eps), rms_norm(k, W("k.norm"), eps)
    if mx.get("rot"):
        pos = np.arange(T)
        q, k = rotate(q, pos, mx["rot"]), rotate(k, pos, mx["rot"])
    q, k, v = rnd(q), rnd(k), rnd(v)
    out = np.zeros((T, H, V), dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        out[:, n] = attend(q[:, n], k[:, g], v[:, g], mx["scale"], (mx.get("mask") or {}).get("size", 0), mx.get("softcap", 0.0),
                           W("sink")[n] if has("sink") else None, rnd)
    if has("g"):
        out = out * sigmoid(h @ W("g").T)[:, :, None]
    return out.reshape(T, H * V)


def linear_attention(q, k, v, decay, state=None):
    """S <- decay S + k v^T, o = S^T q per head. q, k [T, H, D], v [T, H, V]; returns (o, S)."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), dtype=q.dtype) if state is None else state.copy()
    out = np.zeros((T, H, v.shape[2]), dtype=q.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def lightning_mixer(h, mx, W, eps, rnd=exact):
    h = rnd(h)
    T, H, D, V = h.shape[0], mx["heads"], mx["dim"], mx["vdim"]
    q, k = (rnd(silu(h @ W(n).T)).reshape(T, H, D) for n in ("q", "k"))
    v = rnd(silu(h @ W("v").T)).reshape(T, H, V)
    o, _ = linear_attention(q, k, v, np.asarray(mx["decay"], dtype=h.dtype))
    return rms_norm(o.reshape(T, H * V), W("norm"), eps) * sigmoid(h @ W("g").T)


def mixer(h, L, W, has, eps, rnd=exact):
    kind, mx = L["type"].split("_")[0], L["mixer"]
    if kind == "attention":
        return rnd(attention_mixer(h, mx, W, has, eps, rnd)) @ W("o").T
    if kind != "parallel":
        raise ValueError(kind)

    def side(name):
        return (lambda n: W(f"{name}.{n}")), (lambda n: has(f"{name}.{n}"))
    wl, hl = side("left")
    wr, _ = side("right")
    left = rnd(attention_mixer(h, mx["left"], wl, hl, eps, rnd)) @ wl("o").T
    right = rnd(lightning_mixer(h, mx["right"], wr, eps, rnd)) @ wr("o").T
    return mx["left_scale"] * left + mx["right_scale"] * right


def dense_ff(h, W, rnd=exact):
    return rnd(gelu_tanh(rnd(h) @ W("up").T)) @ W("down").T


def layer(x, L, W, has, eps, mult, rnd=exact):
    """Mixer and feed-forward side by side, each behind a norm of its own. W(suffix), has(suffix): the layer's tensors."""
    y = mixer(rms_norm(x, W("norm1"), eps), L, lambda n: W("mix." + n), lambda n: has("mix." + n), eps, rnd)
    if L.get("mlp"):
        y = y + dense_ff(rms_norm(x, W("norm2"), eps), lambda n: W("mlp." + n), rnd)
    return x + mult * y


def schedule(cfg):
    """(layer, first of a pass) in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, i == a) for _ in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


def forward(model, tokens, dtype=np.float64, layers_out=None, rnd=exact):
    """Logits [T, vocab] of a whole sequence; `layers_out` collects the residual stream after every layer run."""
    cfg, t = model["config"], model["tensors"]

    def get(name):
        return np.asarray(t[name], dtype=dtype)
    eps = cfg["norm"]["eps"]
    x0 = get("embed")[np.asarray(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)
    x = x0
    for i, first in schedule(cfg):
        if first:
            x = rnd(np.concatenate([x, x0], axis=-1)) @ get("loop.in").T
        x = layer(x, cfg["layers"][i], lambda n, i=i: get(f"l{i}.{n}"), lambda n, i=i: f"l{i}.{n}" in t, eps, cfg.get("residual_mult", 1.0), rnd)
        if layers_out is not None:
            layers_out.append(x.copy())
    logits = rnd(rms_norm(x, get("final.norm"), eps)) @ get("head").T
    cap = cfg.get("logit_softcap", 0.0)
    return softcap(logits, cap) if cap else logits
