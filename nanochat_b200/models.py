"""Model registry: which class serves a model folder (config.json + model.safetensors).

``config.json`` names the class in ``architecture``.  A registered class offers
``from_dict(config, tensors, dtype, device)`` and, on its instances, ``config``, ``get_device()``,
``make_cache(batch_size, seq_len, ...)`` and ``forward(ids, kv_cache=...)``.
"""
import importlib
import json
import os

import torch

from .weights import read_safetensors

_REGISTRY = {}
_MODULES = ("gpt", "sipadra", "zuvulorn")  # imported on first use; each registers its classes


def register(name):
    def add(cls):
        _REGISTRY[name] = cls
        return cls
    return add


def architectures():
    for m in _MODULES:
        importlib.import_module("." + m, __package__)
    return dict(_REGISTRY)


def model_class(name):
    found = architectures()
    if name not in found:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(found))}")
    return found[name]


def load_model(path, dtype=torch.bfloat16, device="cuda"):
    """The model in folder ``path``, its weights in ``dtype`` on ``device``."""
    with open(os.path.join(path, "config.json")) as f:
        config = json.load(f)
    cls = model_class(config.get("architecture"))
    device = torch.device(device)
    if device.type == "cuda" and device.index is None:
        device = torch.device("cuda", torch.cuda.current_device())
    return cls.from_dict(config, read_safetensors(os.path.join(path, "model.safetensors")), dtype, device)
