"""Virolorn: configuration and weights of the decoder that mixes lightning attention, a gated delta rule with a decay per key
channel and latent attention, for the layer-by-layer runner (``StackModel``).

``stack_config`` turns a config.json into the runner's description; every size and constant comes from there, except the
inner sizes of the delta rule's low-rank decay and gate, which only the tensors' shapes give.  What the design itself
fixes: a norm before and after each sublayer, the convolutions of the delta rule feed silu, one sigmoid gate per head in
latent attention, the feed-forward uses silu, the head is the embedding table.
"""
from __future__ import annotations

from typing import Callable, List, Optional, Tuple

from . import _lib as L
from . import stack as st
from .stack import ConfigError

ARCHITECTURE = "Virolorn"


def _positive(where: str, **sizes):
    for name, v in sizes.items():
        if not isinstance(v, int) or isinstance(v, bool) or v < 1:
            raise ConfigError(f"{where}: {name} {v!r} is not a positive number")


def _lightning(m: dict, where: str) -> dict:
    dim, decay, heads = st.need(m, where, "dim", "decay", "heads")
    _positive(where, dim=dim)
    if len(decay) != heads:
        raise ConfigError(f"{where}: {len(decay)} decays for {heads} heads")
    if not all(0.0 <= d <= 1.0 for d in decay):
        raise ConfigError(f"{where}: decays lie between 0 and 1")
    return {"mixer": L.MIXER_LIGHTNING, "dim": dim, "decay": [float(d) for d in decay]}


def _channel_delta(m: dict, where: str) -> dict:
    kv_heads, dim, conv = st.need(m, where, "kv_heads", "dim", "conv")
    _positive(where, kv_heads=kv_heads, dim=dim, conv=conv)
    return {"mixer": L.MIXER_DELTA, "kv_heads": kv_heads, "dim": dim, "conv_taps": conv}


def _latent_attention(m: dict, where: str) -> dict:
    dim, rot_dim, kv_rank, q_rank, scale, rot = st.need(m, where, "dim", "rot_dim", "kv_rank", "q_rank", "scale", "rot")
    base, dims = st.need(rot, where + " rot", "base", "dims")
    _positive(where, dim=dim, rot_dim=rot_dim, kv_rank=kv_rank, q_rank=q_rank)
    if dims != rot_dim or dims % 2:
        raise ConfigError(f"{where}: {dims} rotated dimensions of {rot_dim}; an even number that equals rot_dim is expected")
    return {"mixer": L.MIXER_LATENT, "dim": dim, "rot_dim": rot_dim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale, "rot_base": base, "head_gate": 1}


MIXERS = {"lightning": _lightning, "channel_delta": _channel_delta, "latent_attention": _latent_attention}


def _owner(entries: List[dict], index: int) -> int:
    """The layer whose tensors layer ``index`` uses (itself, unless 'weights_of' names another)."""
    seen, i = {index}, index
    while entries[i].get("weights_of") is not None:
        i = entries[i]["weights_of"]
        if not isinstance(i, int) or not 0 <= i < len(entries) or i in seen:
            raise ConfigError(f"layer {index}: weights_of does not lead to a layer with tensors")
        seen.add(i)
    return i


def layer_config(entries: List[dict], index: int, shape: Callable[[str], Optional[Tuple[int, ...]]]) -> dict:
    """Entry ``index`` of config 'layers' -> the fields of dp_layer_cfg.  ``shape(name)``: a tensor's shape."""
    where, entry = f"layer {index}", entries[index]
    owner = _owner(entries, index)
    if owner != index and {k: v for k, v in entry.items() if k != "weights_of"} != {k: v for k, v in entries[owner].items() if k != "weights_of"}:
        raise ConfigError(f"{where}: uses the weights of layer {owner} but differs from it")
    kind, m = st.need(entry, where, "type", "mixer")
    if kind not in MIXERS:
        raise ConfigError(f"{where}: unknown type '{kind}'")
    heads, vdim = st.need(m, where, "heads", "vdim")
    _positive(where, heads=heads, vdim=vdim)
    out = {"heads": heads, "vdim": vdim, **MIXERS[kind](m, where)}
    if kind == "channel_delta":
        for field, name in (("decay_rank", "a1"), ("gate_rank", "g1")):
            s = shape(f"l{owner}.mix.{name}")
            if s is None or len(s) != 2:
                raise ConfigError(f"{where}: no matrix l{owner}.mix.{name} to take a size from")
            out[field] = int(s[0])
    mlp = entry.get("mlp")
    if mlp is not None:
        if mlp.get("kind") != "dense":
            raise ConfigError(f"{where}: unknown feed-forward '{mlp.get('kind')}'")
        ff, = st.need(mlp, where + " mlp", "ff")
        _positive(where + " mlp", ff=ff)
        out.update(ff=ff, ff_limit=0.0, ff_slope=1.0, ff_shift=0.0)
    if owner != index:
        out["share"] = owner + 1
    return out


def stack_config(config: dict, shape: Callable[[str], Optional[Tuple[int, ...]]]) -> Tuple[dict, List[dict]]:
    """config.json and the shapes of its tensors -> (stack fields, layer fields)."""
    if config.get("architecture") != ARCHITECTURE:
        raise ConfigError(f"architecture '{config.get('architecture')}' is not {ARCHITECTURE}")
    width, vocab, norm, mult, layers = st.need(config, "config", "width", "vocab", "norm", "residual_mult", "layers")
    eps, = st.need(norm, "norm", "eps")
    _positive("config", width=width, vocab=vocab)
    if not mult:
        raise ConfigError("config: residual_mult 0")
    fields = {"width": width, "vocab": vocab, "streams": 1, "norm_groups": 1, "input_taps": 0, "eps": eps, "embed_scale": 1.0, "post_norm": 1,
              "residual_mult": mult}
    return fields, [layer_config(layers, i, shape) for i in range(len(layers))]


def layer_tensors(layer: dict) -> List[Tuple[str, int]]:
    """(name behind 'l<i>.', tensor id) of every tensor of a layer."""
    if layer.get("share"):
        return []
    names = [("norm1", L.T_NORM1), ("norm1b", L.T_NORM1B), ("mix.o", L.T_O)]
    if layer["mixer"] == L.MIXER_LIGHTNING:
        names += [("mix.q", L.T_Q), ("mix.k", L.T_K), ("mix.v", L.T_V), ("mix.g", L.T_GATE), ("mix.norm", L.T_MIX_NORM)]
    elif layer["mixer"] == L.MIXER_DELTA:
        names += [("mix.q", L.T_Q), ("mix.k", L.T_K), ("mix.v", L.T_V), ("mix.q.conv", L.T_CONV_Q), ("mix.k.conv", L.T_CONV_K), ("mix.v.conv", L.T_CONV_V),
                  ("mix.b", L.T_BETA), ("mix.A_log", L.T_A_LOG), ("mix.dt_bias", L.T_DT_BIAS), ("mix.a1", L.T_A1), ("mix.a2", L.T_A2), ("mix.g1", L.T_G1),
                  ("mix.g2", L.T_G2), ("mix.norm", L.T_MIX_NORM)]
    else:
        names += [("mix.dq", L.T_DQ), ("mix.dq.norm", L.T_DQ_NORM), ("mix.uq", L.T_UQ), ("mix.dkv", L.T_DKV), ("mix.dkv.norm", L.T_DKV_NORM),
                  ("mix.uk", L.T_UK), ("mix.uv", L.T_UV), ("mix.g", L.T_GATE_HEADS)]
    if layer.get("ff"):
        names += [("norm2", L.T_NORM2), ("norm2b", L.T_NORM2B), ("mlp.gate", L.T_FF_GATE), ("mlp.up", L.T_FF_UP), ("mlp.down", L.T_FF_DOWN)]
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
    """The description of the model in a folder (its weight file gives some sizes)."""
    weights = st.open_weights(path)
    try:
        return stack_config(config, weights.shape)
    finally:
        weights.close()


def load(device, path: str, config: dict, max_seq: int, max_batch: int = 1, dtype: str = "bfloat16", max_rows: int = 0):
    """Open a model folder (config.json already read) and upload it."""
    weights = st.open_weights(path)
    try:
        fields, layers = stack_config(config, weights.shape)
        return st.load(device, weights, fields, layers, model_tensors(layers), max_seq, max_batch, dtype, max_rows)
    finally:
        weights.close()
