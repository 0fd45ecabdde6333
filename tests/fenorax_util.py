"""Test helper: small Fenorax configurations and random weights (bfloat16 values, so the oracle and the library see the
same numbers)."""
import numpy as np

from doppler_b200.safetensors import bf16_bits, bf16_values


def mamba(heads=4, vdim=16, state=16, groups=2, conv=4, norm_groups=2, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "conv": conv, "norm_groups": norm_groups}, "mlp": mlp}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, scale=0.4, chunk=13, mlp="default"):
    mlp = {"kind": "dense", "ff": 40, "limit": 0.75} if mlp == "default" else mlp
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": chunk}}, "mlp": mlp}


def config(layers, width=64, vocab=97, streams=3, taps=3, groups=2, eps=1e-4, embed_scale=0.8):
    return {"architecture": "Fenorax", "width": width, "vocab": vocab, "streams": streams, "canon": {"taps": taps}, "norm": {"groups": groups, "eps": eps},
            "embedding": {"scale": embed_scale}, "layers": layers}


def weights(cfg, seed=1):
    """name -> bfloat16 bits"""
    rng = np.random.default_rng(seed)
    W, S, taps = cfg["width"], cfg["streams"], cfg["canon"]["taps"]
    out = {}

    def put(name, a):
        out[name] = bf16_bits(np.asarray(a, np.float32))

    def lin(name, n, k, gain=1.0):
        put(name, rng.standard_normal((n, k)) * gain / np.sqrt(k))

    def near_one(name, n):
        put(name, 1.0 + 0.3 * rng.standard_normal(n))

    put("embed", rng.standard_normal((cfg["vocab"], W)))
    near_one("final.norm", W)
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        for q in ("1", "2") if layer["mlp"] else ("1",):
            near_one(p + "norm" + q, W)
            put(p + "canon" + q, rng.standard_normal((W, taps)) * 0.5)
            put(p + f"hc{q}.in", rng.uniform(0.2, 0.9, S))
            put(p + f"hc{q}.out", rng.uniform(0.4, 1.2, S))
            put(p + f"hc{q}.mix", np.eye(S) * 0.7 + rng.uniform(-0.2, 0.3, (S, S)))
        inner = m["heads"] * m["vdim"]
        lin(p + "mix.o", W, inner, 1.5)
        if layer["type"] == "mamba2":
            ch = inner + 2 * m["groups"] * m["state"]
            lin(p + "mix.in", inner + ch + m["heads"], W, 1.5)
            put(p + "mix.conv", rng.standard_normal((ch, m["conv"])) * 0.7)
            put(p + "mix.conv.b", rng.standard_normal(ch) * 0.3)
            put(p + "mix.dt_bias", rng.uniform(-2.5, 0.5, m["heads"]))
            put(p + "mix.A_log", rng.uniform(-2.5, 1.0, m["heads"]))
            put(p + "mix.D", rng.standard_normal(m["heads"]))
            near_one(p + "mix.norm", inner)
        else:
            lin(p + "mix.q", m["heads"] * m["dim"], W)
            lin(p + "mix.k", m["kv_heads"] * m["dim"], W)
            lin(p + "mix.v", m["kv_heads"] * m["vdim"], W, 1.5)
            lin(p + "mix.g", m["heads"], W, 2.0)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            lin(p + "mlp.gate", ff, W, 1.5)
            lin(p + "mlp.up", ff, W, 1.5)
            lin(p + "mlp.down", W, ff, 1.5)
    return out


def values(w):
    return {k: bf16_values(v).reshape(v.shape).astype(np.float64) for k, v in w.items()}


def build(dev, cfg, w, max_seq, max_batch=1, dtype="float32", max_rows=0):
    from doppler_b200 import fenorax
    from doppler_b200.model import StackModel

    stack, layers = fenorax.stack_config(cfg)
    m = StackModel(dev, stack, layers, max_seq, max_batch, dtype, max_rows)
    fenorax.load_weights(m, w.__getitem__)
    return m


def tokens(cfg, n, seed=0):
    return np.random.default_rng(1000 + seed).integers(0, cfg["vocab"], n).astype(np.int32)


def row_errors(got, want):
    """root mean square error of every row, the mean taken off, relative to the reference's spread"""
    d = np.asarray(got, np.float64) - want
    d -= d.mean(axis=-1, keepdims=True)
    return np.sqrt((d * d).mean(axis=-1)) / want.std()
