"""Small Sofudra models for the tests: configurations, seeded weights, the GPU decoder and the oracle's model."""
import numpy as np

import hybrid_util as U
import kalosm_b200 as kb
from kalosm_b200 import sofudra
from oracle import hybrid as HY
from oracle import sofudra as SO


def rotary(dims=8, base=10000.0, factor=None, original=64, fast=8.0, slow=1.0):
    rot = {"base": base, "dims": dims}
    if factor:
        rot["scaling"] = dict(factor=factor, original=original, fast=fast, slow=slow)
    return rot


def ff(n):
    return {"kind": "dense", "ff": n} if n else None


def attention(heads=6, kv_heads=2, dim=24, vdim=20, window=30, rot=None, scale=None, mlp=56, name="attention"):
    return {"type": name, "mlp": ff(mlp), "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, mask={"size": window},
                                                      rot=rot or rotary(factor=3.0), scale=scale or dim ** -0.5)}


def left(heads=4, kv_heads=2, dim=16, vdim=24, scale=None, softcap=4.0):
    return dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, softcap=softcap)


def right(heads=3, dim=24, vdim=16, decay=None):
    return dict(heads=heads, dim=dim, vdim=vdim, decay=decay or [float(d) for d in np.linspace(0.35, 0.995, heads)])


def parallel(a=None, b=None, left_scale=0.7, right_scale=1.2, mlp=40, name="parallel"):
    return {"type": name, "mlp": ff(mlp), "mixer": dict(left=a or left(), right=b or right(), left_scale=left_scale, right_scale=right_scale)}


def config(layers, width=72, vocab=101, eps=1e-5, loop=None, mult=0.45, embed=3.0, cap=9.0):
    out = {"architecture": "Sofudra", "embedding": {"scale": embed}, "layers": layers, "logit_softcap": cap, "norm": {"eps": eps},
           "residual_mult": mult, "vocab": vocab, "width": width}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def shapes(cfg):
    """{tensor name: shape} of a configuration."""
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "head": (V, E), "final.norm": (E,)}
    if cfg.get("loop"):
        out["loop.in"] = (E, 2 * E)

    def grouped(p, mx, extra):
        H, G, D, N = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
        rows = {"q": H * D, "k": G * D, "v": G * N}
        out.update({p + n: (r, E) for n, r in rows.items()})
        out.update({p + "q.norm": (D,), p + "k.norm": (D,), p + "o": (E, H * N)})
        if extra == "sink":
            out[p + "sink"] = (H,)
        else:
            out.update({p + n + ".b": (r,) for n, r in rows.items()})
            out[p + "g"] = (H, E)
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        out[p + "norm1"] = (E,)
        if L["mlp"]:
            n = L["mlp"]["ff"]
            out.update({p + "norm2": (E,), p + "mlp.up": (n, E), p + "mlp.down": (E, n)})
        if L["type"].startswith("attention"):
            grouped(p + "mix.", mx, "sink")
        else:
            grouped(p + "mix.left.", mx["left"], "bias")
            r = mx["right"]
            hd, hv, p = r["heads"] * r["dim"], r["heads"] * r["vdim"], p + "mix.right."
            out.update({p + "q": (hd, E), p + "k": (hd, E), p + "v": (hv, E), p + "g": (hv, E), p + "o": (E, hv), p + "norm": (hv,)})
    return out


def weights(cfg, seed=0, edit=None):
    """{name: bf16 bits}. Matrices ~ N(0, 1 / columns), embeddings ~ N(0, 1), norms around 1, biases and sinks large enough to show;
    `edit(name, array)` may replace an array."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        w = rng.standard_normal(shape)
        if name.endswith("sink"):
            w = 1.0 + 1.5 * w
        elif name.endswith(".b"):
            w = 0.8 * w
        elif "norm" in name:
            w = 1.0 + 0.2 * w
        elif name != "embed":
            w = w * shape[1] ** -0.5 * 1.3
        if edit:
            new = edit(name, w)
            w = w if new is None else new
        out[name] = U.to_bf16(w)
    return out


def oracle_model(cfg, w):
    return dict(config=cfg, tensors={n: U.from_bf16(b) for n, b in w.items()})


def oracle_logits(cfg, w, tokens, **kw):
    return SO.forward(oracle_model(cfg, w), tokens, **kw)


def gpu_model(dev, cfg, w, dtype, max_seq_len=512, max_batch=1):
    sh = shapes(cfg)
    return sofudra.build(dev, cfg, lambda n: (kb.BF16, sh[n], w[n].view(np.uint8).reshape(-1)), max_seq_len, max_batch, dtype)


def write_checkpoint(folder, cfg, w):
    U.write_checkpoint(folder, cfg, w, shapes(cfg))


def tolerance(cfg, w, tokens, want, dtype):
    """As hybrid_util.tolerance: a fixed bound in 32-bit, three times the effect of rounded operands in bf16."""
    if dtype == "float32":
        return U.TOL[dtype]
    return max(5e-3, 3 * U.err(oracle_logits(cfg, w, tokens, rnd=HY.round_bf16), want))
