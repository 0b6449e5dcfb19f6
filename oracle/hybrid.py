"""Plain, slow restatement of the hybrid decoders (numpy), one function per mechanism.

Test infrastructure: the tests compare the CUDA library with it. Everything is written token by
token from the equations, with no chunking, no caches and no code shared with the product.

A model is a dict {"width", "vocab", "eps", "layers": [...], "tensors": {name: array}} whose layers
are the entries of a checkpoint's config.json ("type", "mixer", "mlp").

`rnd` is the rounding of the operands of matrix products (identity by default): with a 16-bit rounding the
functions show how far rounding alone moves the logits, which is what the tests measure a 16-bit run against.
"""
from __future__ import annotations

import numpy as np


def exact(x):
    return x


def round_bf16(x):
    """To the nearest bf16 (ties to even), in the type of x."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    u = (u + 0x7FFF + ((u >> 16) & 1)) & np.uint32(0xFFFF0000)
    return u.view(np.float32).astype(x.dtype)


def rms_norm(x, w, eps):
    """x / sqrt(mean(x^2) + eps) * w over the last axis."""
    return x / np.sqrt((x * x).mean(-1, keepdims=True) + eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(np.zeros_like(z), z)


def causal_conv(x, w):
    """Depthwise convolution over time: x [T, C], w [C, taps]; the last column meets the current token,
    zeros stand before the start."""
    taps = w.shape[1]
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        for j in range(taps):
            s = t - (taps - 1) + j
            if s >= 0:
                out[t] += w[:, j] * x[s]
    return out


def unit(x):
    """x / sqrt(sum(x^2) + 1e-6) over the last axis."""
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def delta_rule(q, k, v, g, beta, state=None):
    """Gated delta rule. q, k [T, H, D], v [T, H, V], g, beta [T, H]; returns (o [T, H, V], S [H, D, V])."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]), dtype=q.dtype) if state is None else state.copy()
    out = np.zeros_like(v)
    for t in range(T):
        S = S * g[t][:, None, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def delta_mixer(h, mx, W, eps, rnd=exact):
    """The 'delta' mixer over a whole sequence: h [T, width] -> [T, width]. W(name) gives a tensor."""
    h = rnd(h)
    T = h.shape[0]
    H, HK, D, V = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    q, k, v = (silu(causal_conv(h @ W(n).T, W(n + ".conv"))) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, HK, D)) * D ** -0.5
    k = unit(k.reshape(T, HK, D))
    group = np.arange(H) // (H // HK)
    beta = sigmoid(h @ W("b").T)
    g = np.exp(-np.exp(W("A_log")) * softplus(h @ W("a").T + W("dt_bias")))
    o, _ = delta_rule(q[:, group], k[:, group], v.reshape(T, H, V), g, beta)
    o = rms_norm(o, W("norm"), eps) * silu((h @ W("g").T).reshape(T, H, V))
    return rnd(o.reshape(T, H * V)) @ W("o").T


def rotate_half(x, pos, base, dims):
    """Rotary positions on the first `dims` entries of the last axis: entry i pairs with i + dims / 2.
    x [T, ..., n], pos [T]."""
    half = dims // 2
    f = np.asarray(base, dtype=np.float64) ** (-2.0 * np.arange(half) / dims)
    a = (pos[:, None] * f).reshape((x.shape[0],) + (1,) * (x.ndim - 2) + (half,))
    c, s = np.cos(a).astype(x.dtype), np.sin(a).astype(x.dtype)
    u, w = x[..., :half], x[..., half:dims]
    return np.concatenate([u * c - w * s, w * c + u * s, x[..., dims:]], axis=-1)


def latent_rows(h, mx, W, eps, rnd=exact):
    """What a latent-attention layer caches per token: (c [T, kv_rank], rotated key part [T, rot_dim])."""
    r = mx["kv_rank"]
    y = h @ W("dkv").T
    c = rms_norm(y[:, :r], W("dkv.norm"), eps)
    kr = rotate_half(y[:, r:], np.arange(h.shape[0]), mx["rot"]["base"], mx["rot"]["dims"])
    return rnd(c), rnd(kr)


def window_softmax(s, window):
    """Softmax over the visible keys of s [T, T]: query i sees keys j with 0 <= i - j < window."""
    T = s.shape[0]
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    ok = (j <= i) & (i - j < window) if window else (j <= i)
    s = np.where(ok, s, -np.inf)
    p = np.exp(s - s.max(-1, keepdims=True))
    return p / p.sum(-1, keepdims=True)


def latent_mixer(h, mx, W, eps, rows=None, rnd=exact):
    """The 'latent_attention' mixer. `rows` = another layer's (c, rotated key part); returns
    ([T, width], the rows used)."""
    h = rnd(h)
    T = h.shape[0]
    H, D, R, V = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"]
    c, kr = rows if rows is not None else latent_rows(h, mx, W, eps, rnd)
    q = (h @ W("q").T).reshape(T, H, D + R)
    qr = rotate_half(q[..., D:], np.arange(T), mx["rot"]["base"], mx["rot"]["dims"])
    q, qr = rnd(q), rnd(qr)
    k = rnd(c @ W("uk").T).reshape(T, H, D)
    v = rnd(c @ W("uv").T).reshape(T, H, V)
    gate = sigmoid(h @ W("g").T)
    out = np.zeros((T, H, V), dtype=h.dtype)
    window = (mx.get("mask") or {}).get("size", 0)
    for n in range(H):
        s = (q[:, n, :D] @ k[:, n].T + qr[:, n] @ kr.T) * mx["scale"]
        out[:, n] = (rnd(window_softmax(s, window)) @ v[:, n]) * gate[:, n, None]
    return rnd(out.reshape(T, H * V)) @ W("o").T, (c, kr)


def dense_ff(h, W, rnd=exact):
    h = rnd(h)
    return rnd(silu(h @ W("gate").T) * (h @ W("up").T)) @ W("down").T


def forward(model, tokens, dtype=np.float64, layers_out=None, rnd=exact):
    """Logits [T, vocab] of a whole sequence; `layers_out` collects the residual stream per layer."""
    t = model["tensors"]

    def get(name):
        return np.asarray(t[name], dtype=dtype)
    x = get("embed")[np.asarray(tokens)]
    rows = {}
    for i, L in enumerate(model["layers"]):
        h = rms_norm(x, get(f"l{i}.norm1"), model["eps"])
        kind, mx = L["type"].split("_2")[0], L["mixer"]

        def W(n, i=i):
            return get(f"l{i}.mix.{n}")
        if kind == "delta":
            y = delta_mixer(h, mx, W, model["eps"], rnd)
        elif kind == "latent_attention":
            y, rows[i] = latent_mixer(h, mx, W, model["eps"], rows[mx["kv_from"]] if "kv_from" in mx else None, rnd)
        else:
            raise ValueError(kind)
        if L.get("mlp"):
            y = y + dense_ff(h, lambda n, i=i: get(f"l{i}.mlp.{n}"), rnd)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.copy())
    return rnd(rms_norm(x, get("final.norm"), model["eps"])) @ get("head").T
