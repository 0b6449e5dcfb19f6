"""Checkpoint folders of the dense architectures (config.json and model.safetensors): what their loaders share."""
import json
import os
import re

import numpy as np

from .safetensors import SafetensorsFile


class ConfigError(ValueError):
    pass


def mixer_kind(name):
    """The kind of a layer's type: a trailing _<n> only tells apart variants of other sizes."""
    return re.sub(r"_\d+$", "", name)


def open_checkpoint(path, architecture):
    """(config, tensor) of a folder; `tensor(name)` returns (ggml type, shape, bytes)."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    if config.get("architecture") != architecture:
        raise ConfigError(f"architecture {config.get('architecture')!r} is not {architecture!r}")
    return config, SafetensorsFile(os.path.join(path, "model.safetensors")).raw


def fill(model, tensor, names):
    """Sets the model-level tensors and `names`: (library tensor name, entry, checkpoint name)."""
    for short, entry, name in [("token_embd", -1, "embed"), ("output", -1, "head"), ("output_norm", -1, "final.norm")] + list(names):
        ty, shape, raw = tensor(name)
        model.set_tensor(short, entry, ty, shape, np.asarray(raw))
    return model
