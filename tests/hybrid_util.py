"""Small Koludra models for the tests: configurations, seeded weights, the GPU decoder and the oracle's model."""
import json
import os

import numpy as np

import kalosm_b200 as kb
from kalosm_b200 import koludra
from kalosm_b200.safetensors import write_safetensors
from oracle import hybrid as HY


def delta(heads=4, kv_heads=2, dim=24, vdim=40, conv=4, ff=56, name="delta"):
    return {"type": name, "mixer": dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv),
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def latent(heads=3, dim=32, rot=16, vdim=24, rank=40, window=20, base=10000.0, scale=None, kv_from=None, ff=48):
    mx = dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, mask={"size": window},
              rot={"base": base, "dims": rot}, scale=scale or float((dim + rot) ** -0.5))
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mx, "mlp": {"kind": "dense", "ff": ff} if ff else None}


def config(layers, width=72, vocab=101, eps=1e-5):
    return {"architecture": "Koludra", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


def shapes(cfg):
    """{tensor name: shape} of a configuration."""
    E, V = cfg["width"], cfg["vocab"]
    out = {"embed": (V, E), "head": (V, E), "final.norm": (E,)}
    for i, L in enumerate(cfg["layers"]):
        mx, p = L["mixer"], f"l{i}."
        H, hv = mx["heads"], mx["heads"] * mx["vdim"]
        out[p + "norm1"] = (E,)
        if L["mlp"]:
            ff = L["mlp"]["ff"]
            out.update({p + "mlp.gate": (ff, E), p + "mlp.up": (ff, E), p + "mlp.down": (E, ff)})
        out[p + "mix.o"] = (E, hv)
        if L["type"].startswith("delta"):
            qk = mx["kv_heads"] * mx["dim"]
            for n, c in (("q", qk), ("k", qk), ("v", hv)):
                out[p + f"mix.{n}"] = (c, E)
                out[p + f"mix.{n}.conv"] = (c, mx["conv"])
            out.update({p + "mix.b": (H, E), p + "mix.a": (H, E), p + "mix.A_log": (H,), p + "mix.dt_bias": (H,),
                        p + "mix.norm": (mx["vdim"],), p + "mix.g": (hv, E)})
        else:
            out.update({p + "mix.q": (H * (mx["dim"] + mx["rot_dim"]), E), p + "mix.g": (H, E),
                        p + "mix.uk": (H * mx["dim"], mx["kv_rank"]), p + "mix.uv": (hv, mx["kv_rank"])})
            if "kv_from" not in mx:
                out.update({p + "mix.dkv": (mx["kv_rank"] + mx["rot_dim"], E), p + "mix.dkv.norm": (mx["kv_rank"],)})
    return out


def to_bf16(x):
    """f32 -> the bits of the nearest bf16 (ties to even)."""
    u = np.ascontiguousarray(x, dtype=np.float32).view(np.uint32)
    return ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)


def from_bf16(u):
    return (u.astype(np.uint32) << 16).view(np.float32)


def weights(cfg, seed=0, edit=None):
    """{name: bf16 bits}. Matrices ~ N(0, 1 / columns) (embeddings ~ N(0, 1)), norms around 1, decays between slow and
    fast; `edit(name, array)` may replace an array."""
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in shapes(cfg).items():
        if name.endswith("A_log"):
            w = np.log(rng.uniform(0.02, 4.0, shape))
        elif name.endswith("dt_bias"):
            w = rng.uniform(-3.0, 1.0, shape)
        elif name.endswith(".conv"):
            w = rng.standard_normal(shape) * 0.6
        elif "norm" in name:
            w = 1.0 + 0.2 * rng.standard_normal(shape)
        elif name == "embed":
            w = rng.standard_normal(shape)
        else:
            w = rng.standard_normal(shape) * shape[1] ** -0.5 * 1.3
        if edit:
            new = edit(name, w)
            w = w if new is None else new
        out[name] = to_bf16(w)
    return out


def oracle_model(cfg, w):
    return dict(width=cfg["width"], vocab=cfg["vocab"], eps=cfg["norm"]["eps"], layers=cfg["layers"],
                tensors={n: from_bf16(b) for n, b in w.items()})


def gpu_model(dev, cfg, w, dtype, max_seq_len=512, max_batch=1):
    sh = shapes(cfg)
    return koludra.build(dev, cfg, lambda n: (kb.BF16, sh[n], w[n].view(np.uint8).reshape(-1)), max_seq_len, max_batch, dtype)


def write_checkpoint(folder, cfg, w, sh=None):
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    sh = sh or shapes(cfg)
    write_safetensors(os.path.join(folder, "model.safetensors"), [(n, "BF16", sh[n], b) for n, b in w.items()])


def identity_head(cfg):
    """An edit for `weights`: vocab = width and the head is the identity, so that the logits are the normalised
    residual stream itself."""
    def edit(name, w):
        if name == "head":
            return np.eye(cfg["width"])
        if name == "final.norm":
            return np.ones_like(w)
        return None
    return edit


def err(got, want):
    """Root mean square difference of the logits, per position, relative to their overall scale; the worst."""
    want = np.asarray(want, dtype=np.float64)
    d = np.asarray(got, dtype=np.float64) - want
    return float(np.sqrt((d * d).mean(-1)).max() / np.sqrt((want * want).mean()))


TOL = {"float32": 2e-5, "bfloat16": 3e-2}


def tolerance(cfg, w, tokens, want, dtype):
    """float32: a fixed small bound. bfloat16: three times what rounding the operands of the products does to the
    oracle (a sensitive token is sensitive in both), at least 0.5 %."""
    if dtype == "float32":
        return TOL[dtype]
    return max(5e-3, 3 * err(HY.forward(oracle_model(cfg, w), tokens, rnd=HY.round_bf16), want))


def run_portions(m, tokens, sizes, reset=True):
    """Feeds `tokens` in portions of the given sizes (the last one repeats); logits of every position."""
    if reset:
        m.reset()
    out, at, k = [], 0, 0
    while at < len(tokens):
        n = min(sizes[min(k, len(sizes) - 1)], len(tokens) - at)
        m.forward(tokens[at:at + n], want_logits=False)
        out.append(m.logits_at(range(n)))
        at += n
        k += 1
    return np.concatenate(out)


def oracle_logits(cfg, w, tokens):
    return HY.forward(oracle_model(cfg, w), tokens)
