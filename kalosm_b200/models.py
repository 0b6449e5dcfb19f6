"""Model registry: the architecture a checkpoint names decides which loader builds its decoder."""
import json
import os

from . import gguf, koludra, sofudra


def _gguf_llama(device, path, max_seq_len=None, max_batch=1, dtype=None):
    if dtype not in (None, "bfloat16"):
        raise ValueError("quantised Llama checkpoints have one precision (no float32 mode)")
    return gguf.load_llama(device, path, max_seq_len=max_seq_len, max_batch=max_batch)


# architecture name -> loader(device, path, max_seq_len, max_batch, dtype)
REGISTRY = {"llama": _gguf_llama, koludra.ARCHITECTURE: koludra.load, sofudra.ARCHITECTURE: sofudra.load}


# architectures that the dense part of the library serves (build.build(part="dense"))
DENSE = (koludra.ARCHITECTURE, sofudra.ARCHITECTURE)


def architecture(path):
    """The architecture name of a checkpoint: a folder with config.json, or a GGUF file."""
    if os.path.isdir(path):
        with open(os.path.join(path, "config.json")) as f:
            return json.load(f).get("architecture")
    return gguf.GgufFile(path).metadata.get("general.architecture")


def load_model(device, path, max_seq_len=None, max_batch=1, dtype="bfloat16"):
    """Builds the decoder of a checkpoint. `dtype` is the precision of dense models ("bfloat16" or "float32")."""
    name = architecture(path)
    if name not in REGISTRY:
        raise ValueError(f"architecture {name!r} is not supported (known: {', '.join(sorted(REGISTRY))})")
    return REGISTRY[name](device, path, max_seq_len=max_seq_len, max_batch=max_batch, dtype=dtype)
