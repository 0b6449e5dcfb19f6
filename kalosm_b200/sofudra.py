"""Sofudra: a decoder whose layers add a mixer and an ungated feed-forward, each behind a norm of its own, to the residual
stream. The mixer is windowed softmax attention with rotary positions and sinks, or softmax attention over all tokens
beside a linear attention. Some layers run several times. Configuration (config.json) and weights (model.safetensors) of
a checkpoint folder.

config.json: "vocab", "width", "norm": {"eps"}, "embedding": {"scale"}, "residual_mult", "logit_softcap", "loop": {"start",
"stop", "times"} and "layers", each with its mixer's "type", its sizes ("mixer") and its feed-forward ("mlp", or null).
Tensors: "embed", "head", "final.norm", "loop.in" and per layer "l<i>.norm1", "l<i>.norm2", "l<i>.mix.*", "l<i>.mlp.*".
"""
import numpy as np

from . import (ATTN_BIAS, ATTN_GATE, ATTN_QK_NORM, ATTN_SINK, F32, FFN_GELU, MIX_ATTENTION, MIX_LINEAR, HybridDecoder)
from .checkpoint import ConfigError, fill, mixer_kind, open_checkpoint

ARCHITECTURE = "Sofudra"
# what the two attention mixers have beyond their sizes
WINDOWED = ATTN_QK_NORM | ATTN_SINK
BESIDE = ATTN_QK_NORM | ATTN_BIAS | ATTN_GATE
# suffix of a mixer tensor -> the library's tensor name
PROJECTIONS = {"q": "mix_q", "k": "mix_k", "v": "mix_v", "o": "mix_out"}
PARTS = {ATTN_QK_NORM: {"q.norm": "mix_q_norm", "k.norm": "mix_k_norm"}, ATTN_SINK: {"sink": "mix_sink"}, ATTN_GATE: {"g": "mix_gate"},
         ATTN_BIAS: {"q.b": "mix_q_bias", "k.b": "mix_k_bias", "v.b": "mix_v_bias"}}
LINEAR = dict(PROJECTIONS, g="mix_gate", norm="mix_out_norm")


def rotation(index, rot):
    """The LayerConfig fields of a rotation."""
    out = dict(rot_dim=int(rot["dims"]), rope_base=float(rot["base"]))
    scaling = rot.get("scaling")
    if scaling:
        if not float(scaling["factor"]) > 0:
            raise ConfigError(f"layer {index}: rotation scaled by {scaling['factor']}")
        out.update(yarn_factor=float(scaling["factor"]), yarn_fast=float(scaling["fast"]), yarn_slow=float(scaling["slow"]),
                   yarn_original=int(scaling["original"]))
    return out


def attention(index, mx, parts):
    """The LayerConfig fields of a softmax attention."""
    out = dict(mixer=MIX_ATTENTION, heads=int(mx["heads"]), kv_heads=int(mx["kv_heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]),
               scale=float(mx["scale"]), softcap=float(mx.get("softcap") or 0.0), window=int((mx.get("mask") or {}).get("size", 0)), parts=parts)
    if mx.get("rot"):
        out.update(rotation(index, mx["rot"]))
    return out


def layer_entries(index, layer):
    """One entry of config "layers" as [(fields of LayerConfig, {checkpoint suffix: library tensor name}, decays or None)]."""
    kind, mx, mlp = mixer_kind(layer["type"]), layer["mixer"], layer.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ConfigError(f"layer {index}: feed-forward kind {mlp.get('kind')!r} is not supported")
    head, names = {}, {"norm1": "attn_norm"}
    if mlp:
        head = dict(ffn=int(mlp["ff"]), ffn_act=FFN_GELU, two_norms=1)
        names.update({"norm2": "ffn_norm", "mlp.up": "ffn_up", "mlp.down": "ffn_down"})

    def attention_names(prefix, parts):
        out = dict(PROJECTIONS)
        for bit, extra in PARTS.items():
            if parts & bit:
                out.update(extra)
        return {prefix + n: short for n, short in out.items()}
    if kind == "attention":
        return [(dict(attention(index, mx, WINDOWED), **head), dict(names, **attention_names("mix.", WINDOWED)), None)]
    if kind != "parallel":
        raise ConfigError(f"layer {index}: mixer type {layer['type']!r} is not supported")
    left, right = mx["left"], mx["right"]
    decay = [float(d) for d in right["decay"]]
    if len(decay) != int(right["heads"]):
        raise ConfigError(f"layer {index}: {len(decay)} decays for {right['heads']} heads")
    linear = dict(mixer=MIX_LINEAR, beside=1, heads=int(right["heads"]), dim=int(right["dim"]), vdim=int(right["vdim"]),
                  out_scale=float(mx["right_scale"]))
    return [(dict(attention(index, left, BESIDE), out_scale=float(mx["left_scale"]), **head),
             dict(names, **attention_names("mix.left.", BESIDE)), None),
            (linear, {"mix.right." + n: short for n, short in LINEAR.items()}, decay)]


def stack(config):
    """The StackConfig fields of a configuration."""
    loop = config.get("loop") or {}
    return dict(embed_scale=float((config.get("embedding") or {}).get("scale", 1.0)), residual_mult=float(config.get("residual_mult", 1.0)),
                logit_softcap=float(config.get("logit_softcap") or 0.0), loop_start=int(loop.get("start", 0)),
                loop_stop=int(loop.get("stop", 0)), loop_times=int(loop.get("times", 0)))


def build(device, config, tensor, max_seq_len, max_batch=1, dtype="bfloat16"):
    """A decoder from a parsed configuration; `tensor(name)` returns (ggml type, shape, bytes)."""
    entries = [(i, e) for i, layer in enumerate(config["layers"]) for e in layer_entries(i, layer)]
    around = stack(config)
    m = HybridDecoder(device, hidden=int(config["width"]), vocab=int(config["vocab"]), rms_eps=float(config["norm"]["eps"]),
                      layers=[fields for _, (fields, _, _) in entries], stack=around, max_seq_len=max_seq_len, max_batch=max_batch,
                      compute=dtype)
    names = [("loop_in", -1, "loop.in")] if around["loop_times"] else []
    for at, (i, (_, tensors, decay)) in enumerate(entries):
        names += [(short, at, f"l{i}.{suffix}") for suffix, short in tensors.items()]
        if decay is not None:
            m.set_tensor("mix_head_decay", at, F32, (len(decay),), np.asarray(decay, dtype=np.float32))
    return fill(m, tensor, names)


def load(device, path, max_seq_len=None, max_batch=1, dtype="bfloat16"):
    """Loads a checkpoint folder (config.json and model.safetensors)."""
    config, tensor = open_checkpoint(path, ARCHITECTURE)
    return build(device, config, tensor, max_seq_len or 4096, max_batch, dtype)
