"""Fenorax: configuration and weights of the hybrid decoder (Mamba-2 and chunked attention layers over hyper-connected
residual streams), for the layer-by-layer runner (``StackModel``).

``stack_config`` turns a config.json into the runner's description; every size and constant comes from there.  What the
design itself fixes: attention heads are divided by their root mean square without a weight and gated per head, no
rotation, the gated feed-forward uses sigmoid(1.702 g) and u + 1, the head is the embedding table.
"""
from __future__ import annotations

from typing import List, Tuple

from . import _lib as L
from . import stack as st
from .stack import ConfigError

ARCHITECTURE = "Fenorax"
FF_SLOPE, FF_SHIFT = 1.702, 1.0


def layer_config(entry: dict, index: int) -> dict:
    """One entry of config 'layers' -> the fields of dp_layer_cfg."""
    where = f"layer {index}"
    kind, m = st.need(entry, where, "type", "mixer")
    heads, vdim = st.need(m, where, "heads", "vdim")
    out = {"heads": heads, "vdim": vdim}
    if kind == "mamba2":
        state, groups, conv, norm_groups = st.need(m, where, "state", "groups", "conv", "norm_groups")
        out.update(mixer=L.MIXER_MAMBA2, state=state, groups=groups, conv_taps=conv, norm_groups=norm_groups)
    elif kind == "attention":
        kv_heads, dim, scale, mask = st.need(m, where, "kv_heads", "dim", "scale", "mask")
        out.update(mixer=L.MIXER_ATTENTION, kv_heads=kv_heads, dim=dim, scale=scale, chunk=st.need(mask, where + " mask", "size")[0], unit_rms_qk=1, head_gate=1)
    else:
        raise ConfigError(f"{where}: unknown type '{kind}'")
    mlp = entry.get("mlp")
    if mlp is not None:
        if mlp.get("kind") != "dense":
            raise ConfigError(f"{where}: unknown feed-forward '{mlp.get('kind')}'")
        ff, limit = st.need(mlp, where + " mlp", "ff", "limit")
        if not limit > 0:
            raise ConfigError(f"{where}: feed-forward limit {limit} must be positive")
        out.update(ff=ff, ff_limit=limit, ff_slope=FF_SLOPE, ff_shift=FF_SHIFT)
    return out


def stack_config(config: dict) -> Tuple[dict, List[dict]]:
    """config.json -> (stack fields, layer fields)."""
    if config.get("architecture") != ARCHITECTURE:
        raise ConfigError(f"architecture '{config.get('architecture')}' is not {ARCHITECTURE}")
    width, vocab, streams, norm, canon, embedding, layers = st.need(config, "config", "width", "vocab", "streams", "norm", "canon", "embedding", "layers")
    eps, groups = st.need(norm, "norm", "eps", "groups")
    stack = {"width": width, "vocab": vocab, "streams": streams, "norm_groups": groups, "input_taps": st.need(canon, "canon", "taps")[0], "eps": eps,
             "embed_scale": st.need(embedding, "embedding", "scale")[0]}
    return stack, [layer_config(e, i) for i, e in enumerate(layers)]


def layer_tensors(layer: dict) -> List[Tuple[str, int]]:
    """(name behind 'l<i>.', tensor id) of every tensor of a layer."""
    names = [("norm1", L.T_NORM1), ("canon1", L.T_CONV1), ("hc1.in", L.T_HC1_IN), ("hc1.out", L.T_HC1_OUT), ("hc1.mix", L.T_HC1_MIX), ("mix.o", L.T_O)]
    if layer["mixer"] == L.MIXER_MAMBA2:
        names += [("mix.in", L.T_SSM_IN), ("mix.conv", L.T_SSM_CONV), ("mix.conv.b", L.T_SSM_CONV_B), ("mix.dt_bias", L.T_SSM_DT_BIAS),
                  ("mix.A_log", L.T_SSM_A_LOG), ("mix.D", L.T_SSM_D), ("mix.norm", L.T_SSM_NORM)]
    else:
        names += [("mix.q", L.T_Q), ("mix.k", L.T_K), ("mix.v", L.T_V), ("mix.g", L.T_GATE_HEADS)]
    if layer.get("ff"):
        names += [("norm2", L.T_NORM2), ("canon2", L.T_CONV2), ("hc2.in", L.T_HC2_IN), ("hc2.out", L.T_HC2_OUT), ("hc2.mix", L.T_HC2_MIX),
                  ("mlp.gate", L.T_FF_GATE), ("mlp.up", L.T_FF_UP), ("mlp.down", L.T_FF_DOWN)]
    return names


def model_tensors(layers: List[dict]) -> List[Tuple[str, int, int]]:
    """(full name, layer or -1, tensor id) of every tensor of a model."""
    out = [("embed", -1, L.T_EMBED), ("final.norm", -1, L.T_FINAL_NORM)]
    for i, layer in enumerate(layers):
        out += [(f"l{i}.{name}", i, tid) for name, tid in layer_tensors(layer)]
    return out


def load_weights(model, get):
    """Upload every tensor of the model; ``get(name)`` returns its bfloat16 bits."""
    st.load_tensors(model, model_tensors(model.layers), get)


def describe(path: str, config: dict) -> Tuple[dict, List[dict]]:
    """The description of the model in a folder."""
    return stack_config(config)


def load(device, path: str, config: dict, max_seq: int, max_batch: int = 1, dtype: str = "bfloat16", max_rows: int = 0):
    """Open a model folder (config.json already read) and upload it."""
    fields, layers = stack_config(config)
    weights = st.open_weights(path)
    try:
        return st.load(device, weights, fields, layers, model_tensors(layers), max_seq, max_batch, dtype, max_rows)
    finally:
        weights.close()
