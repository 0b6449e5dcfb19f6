"""Koludra: a decoder whose layers are gated delta rules or latent attention beside a gated feed-forward,
both reading one norm. Configuration (config.json) and weights (model.safetensors) of a checkpoint folder.

config.json: "vocab", "width", "norm": {"eps"} and "layers", each with its mixer's "type", its sizes
("mixer") and its feed-forward ("mlp", or null). Tensors: "embed", "head", "final.norm" and per layer
"l<i>.norm1", "l<i>.mix.*", "l<i>.mlp.*".
"""
from . import MIX_DELTA, MIX_LATENT, HybridDecoder
from .checkpoint import ConfigError, fill, mixer_kind, open_checkpoint

ARCHITECTURE = "Koludra"
# suffix of a layer tensor -> the library's tensor name
COMMON = {"norm1": "attn_norm", "mix.q": "mix_q", "mix.g": "mix_gate", "mix.o": "mix_out"}
FFN = {"mlp.gate": "ffn_gate", "mlp.up": "ffn_up", "mlp.down": "ffn_down"}
DELTA = {"mix.k": "mix_k", "mix.v": "mix_v", "mix.b": "mix_beta", "mix.a": "mix_decay", "mix.q.conv": "mix_q_conv",
         "mix.k.conv": "mix_k_conv", "mix.v.conv": "mix_v_conv", "mix.A_log": "mix_a_log", "mix.dt_bias": "mix_dt_bias",
         "mix.norm": "mix_out_norm"}
LATENT = {"mix.uk": "mix_uk", "mix.uv": "mix_uv"}
LATENT_OWN = {"mix.dkv": "mix_dkv", "mix.dkv.norm": "mix_dkv_norm"}


def layer_config(index, layer):
    """One entry of config "layers" as the fields of LayerConfig."""
    kind, mx, mlp = mixer_kind(layer["type"]), layer["mixer"], layer.get("mlp")
    if mlp is not None and mlp.get("kind") != "dense":
        raise ConfigError(f"layer {index}: feed-forward kind {mlp.get('kind')!r} is not supported")
    out = dict(ffn=int(mlp["ff"]) if mlp else 0, heads=int(mx["heads"]), dim=int(mx["dim"]), vdim=int(mx["vdim"]))
    if kind == "delta":
        return dict(out, mixer=MIX_DELTA, kv_heads=int(mx["kv_heads"]), conv=int(mx["conv"]))
    if kind != "latent_attention":
        raise ConfigError(f"layer {index}: mixer type {layer['type']!r} is not supported")
    rot, mask = mx["rot"], mx.get("mask") or {}
    if int(rot["dims"]) != int(mx["rot_dim"]):
        raise ConfigError(f"layer {index}: rot.dims {rot['dims']} differs from rot_dim {mx['rot_dim']}")
    return dict(out, mixer=MIX_LATENT, kv_rank=int(mx["kv_rank"]), rot_dim=int(mx["rot_dim"]), window=int(mask.get("size", 0)),
                kv_from=int(mx.get("kv_from", -1)), rope_base=float(rot["base"]), scale=float(mx["scale"]))


def layer_tensors(layer):
    """{checkpoint suffix: library tensor name} of one entry of config "layers"."""
    names = dict(COMMON)
    if layer.get("mlp"):
        names.update(FFN)
    if mixer_kind(layer["type"]) == "delta":
        names.update(DELTA)
    else:
        names.update(LATENT)
        if "kv_from" not in layer["mixer"]:
            names.update(LATENT_OWN)
    return names


def build(device, config, tensor, max_seq_len, max_batch=1, dtype="bfloat16"):
    """A decoder from a parsed configuration; `tensor(name)` returns (ggml type, shape, bytes)."""
    m = HybridDecoder(device, hidden=int(config["width"]), vocab=int(config["vocab"]), rms_eps=float(config["norm"]["eps"]),
                      layers=[layer_config(i, layer) for i, layer in enumerate(config["layers"])], max_seq_len=max_seq_len,
                      max_batch=max_batch, compute=dtype)
    return fill(m, tensor, [(short, i, f"l{i}.{suffix}") for i, layer in enumerate(config["layers"])
                            for suffix, short in layer_tensors(layer).items()])


def load(device, path, max_seq_len=None, max_batch=1, dtype="bfloat16"):
    """Loads a checkpoint folder (config.json and model.safetensors)."""
    config, tensor = open_checkpoint(path, ARCHITECTURE)
    return build(device, config, tensor, max_seq_len or 4096, max_batch, dtype)
