"""Model registry: which loader opens a model folder.

A folder with ``manifest.json`` is an RDRR artifact of the dense Q4_K decoder; one with ``config.json`` names its
architecture there.  ``load_model`` returns a runner (:mod:`doppler_b200.model`), the same calls whatever the model.
"""
from __future__ import annotations

import json
import os
from types import ModuleType
from typing import Dict

from . import fenorax, virolorn

DTYPES = ("bfloat16", "float32")


class UnknownModel(Exception):
    pass


# architecture named by config.json -> the design's module: describe(path, config) and
# load(device, path, config, max_seq, max_batch, dtype, max_rows)
ARCHITECTURES: Dict[str, ModuleType] = {m.ARCHITECTURE: m for m in (fenorax, virolorn)}


def describe(path: str) -> dict:
    """{"kind": "rdrr"} or {"kind": architecture, "config": config.json}; raises UnknownModel."""
    if os.path.exists(os.path.join(path, "manifest.json")):
        return {"kind": "rdrr"}
    cfg = os.path.join(path, "config.json")
    if not os.path.exists(cfg):
        raise UnknownModel(f"{path}: neither manifest.json nor config.json")
    with open(cfg) as f:
        config = json.load(f)
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise UnknownModel(f"{path}: architecture '{name}' (known: {', '.join(sorted(ARCHITECTURES))})")
    return {"kind": name, "config": config}


def load_model(device, path: str, max_seq: int, max_batch: int = 1, dtype: str = "bfloat16", max_rows: int = 0):
    """Open the model in folder ``path``.  ``dtype`` and ``max_rows`` (rows of one block of a prompt) concern the
    architectures of ``config.json``; the Q4_K decoder has one precision (f32 activations)."""
    if dtype not in DTYPES:
        raise ValueError(f"dtype '{dtype}' (one of {', '.join(DTYPES)})")
    d = describe(path)
    if d["kind"] == "rdrr":
        from .rdrr import load_decoder

        return load_decoder(device, path, max_seq, max_batch)
    return ARCHITECTURES[d["kind"]].load(device, path, d["config"], max_seq, max_batch, dtype, max_rows)
