"""What the designs of the layer-by-layer runner (``StackModel``) share: reading their config.json and their weight file.

A design module supplies ``stack_config(config[, shape])`` (config.json -> the fields of dp_stack_cfg and dp_layer_cfg) and
``model_tensors(layers)`` (tensor names of its weight file -> the runner's tensor ids).
"""
from __future__ import annotations

import os
from typing import Callable, List, Tuple

from .safetensors import SafetensorsFile

WEIGHTS_FILE = "model.safetensors"


class ConfigError(Exception):
    pass


def need(d: dict, where: str, *keys):
    missing = [k for k in keys if k not in d]
    if missing:
        raise ConfigError(f"{where}: missing {', '.join(missing)}")
    return [d[k] for k in keys]


def load_tensors(model, names: List[Tuple[str, int, int]], get: Callable):
    """Upload the tensors (name, layer or -1, tensor id); ``get(name)`` returns bfloat16 bits."""
    for name, layer, tid in names:
        model.load_tensor(layer, tid, get(name))


def open_weights(path: str) -> SafetensorsFile:
    return SafetensorsFile(os.path.join(path, WEIGHTS_FILE))


def load(device, weights: SafetensorsFile, stack: dict, layers: List[dict], names: List[Tuple[str, int, int]], max_seq: int, max_batch: int, dtype: str,
         max_rows: int):
    """A runner of the described model with the weights of an open file."""
    from .model import StackModel  # needs the CUDA library

    def get(name):
        if name in weights and weights.dtype(name) != "BF16":
            raise ConfigError(f"{name}: dtype {weights.dtype(name)}, expected BF16")
        return weights.tensor(name)

    model = StackModel(device, stack, layers, max_seq, max_batch, dtype, max_rows)
    try:
        load_tensors(model, names, get)
    except Exception:
        model.destroy()
        raise
    return model
