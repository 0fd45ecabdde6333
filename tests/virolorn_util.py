"""Test helper: small Virolorn configurations and random weights (bfloat16 values, so the oracle and the library see the same
numbers)."""
import numpy as np

from doppler_b200.safetensors import bf16_bits
from fenorax_util import row_errors, tokens, values  # noqa: F401  (the same for every design)

FF = {"kind": "dense", "ff": 40}


def lightning(heads=3, dim=20, vdim=12, decay=None, mlp=None):
    decay = [float(d) for d in np.linspace(0.55, 0.97, heads)] if decay is None else decay
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay}, "mlp": mlp}


def delta(heads=4, kv_heads=2, dim=20, vdim=12, conv=4, mlp=None, ranks=(6, 10)):
    return {"type": "channel_delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}, "mlp": mlp, "_ranks": ranks}


def latent(heads=3, dim=24, rot_dim=8, vdim=20, kv_rank=40, q_rank=24, scale=0.35, base=50.0, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale,
                      "rot": {"base": base, "dims": rot_dim}}}


def config(layers, width=64, vocab=97, eps=1e-4, mult=0.7):
    """Layers may be the builders' entries or ("again", j): layer j's weights once more."""
    out = []
    for e in layers:
        out.append(dict(out[e[1]], weights_of=e[1]) if isinstance(e, tuple) else e)
    return {"architecture": "Virolorn", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": out}


def public(cfg):
    """What a config.json holds: without the inner sizes that only the tensors' shapes give."""
    return dict(cfg, layers=[{k: v for k, v in e.items() if k != "_ranks"} for e in cfg["layers"]])


def weights(cfg, seed=1):
    """name -> bfloat16 bits"""
    rng = np.random.default_rng(seed)
    W = cfg["width"]
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
        if "weights_of" in layer:
            continue
        m, p = layer["mixer"], f"l{i}."
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if layer["mlp"] else ()):
            near_one(p + n, W)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        lin(p + "mix.o", W, H * V)
        if layer["type"] == "lightning":
            for t, n in (("q", H * D), ("k", H * D), ("v", H * V), ("g", H * V)):
                lin(p + "mix." + t, n, W, 1.5)
            near_one(p + "mix.norm", H * V)
        elif layer["type"] == "channel_delta":
            QK, taps, (ra, rg) = m["kv_heads"] * D, m["conv"], layer["_ranks"]
            for t, n in (("q", QK), ("k", QK), ("v", H * V)):
                lin(p + "mix." + t, n, W, 1.5)
                put(p + f"mix.{t}.conv", rng.standard_normal((n, taps)) * 0.7)
            lin(p + "mix.b", H, W, 1.5)
            put(p + "mix.A_log", rng.uniform(-3.0, 1.0, H))
            put(p + "mix.dt_bias", rng.uniform(-3.0, 0.5, H * D))
            lin(p + "mix.a1", ra, W)
            lin(p + "mix.a2", H * D, ra, 1.5)
            lin(p + "mix.g1", rg, W)
            lin(p + "mix.g2", H * V, rg, 2.0)
            near_one(p + "mix.norm", V)
        else:
            R, K, Q = m["rot_dim"], m["kv_rank"], m["q_rank"]
            lin(p + "mix.dq", Q, W)
            near_one(p + "mix.dq.norm", Q)
            lin(p + "mix.uq", H * (D + R), Q, 1.5)
            lin(p + "mix.dkv", K + R, W, 1.5)
            near_one(p + "mix.dkv.norm", K)
            lin(p + "mix.uk", H * D, K, 1.5)
            lin(p + "mix.uv", H * V, K, 1.5)
            lin(p + "mix.g", H, W, 2.0)
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            lin(p + "mlp.gate", ff, W, 1.5)
            lin(p + "mlp.up", ff, W, 1.5)
            lin(p + "mlp.down", W, ff)
    return out


def build(dev, cfg, w, max_seq, max_batch=1, dtype="float32", max_rows=0):
    from doppler_b200 import virolorn
    from doppler_b200.model import StackModel

    stack, layers = virolorn.stack_config(public(cfg), lambda n: w[n].shape if n in w else None)
    m = StackModel(dev, stack, layers, max_seq, max_batch, dtype, max_rows)
    virolorn.load_weights(m, w.__getitem__)
    return m


def far_key_model(heads=2, dim=16, rot_dim=4, vdim=16, kv_rank=16, q_rank=8, scale=3.0, mult=1.0):
    """One latent-attention layer in which token 1's key stands out for every query and its value is large: rows 0 of the
    latents carry a query direction that all tokens share and a key direction that only token 1 has."""
    rng = np.random.default_rng(7)
    W, vocab = 48, 40
    cfg = config([latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=1e4)], width=W, vocab=vocab, mult=mult)
    w = values(weights(cfg, 3))
    e = rng.standard_normal((vocab, W)) * 0.3
    e[:, 0] = 2.0
    e[:, 1] = -1.0
    e[1, 1] = 3.0
    e[1, 2:] = rng.standard_normal(W - 2)
    w["embed"] = e
    w["l0.norm1"] = np.ones(W)
    dq, dkv = 0.05 * rng.standard_normal((q_rank, W)), 0.3 * rng.standard_normal((kv_rank + rot_dim, W)) / np.sqrt(W)
    dq[0, 0], dkv[0, 1] = 1.0, 1.0
    dkv[kv_rank:] *= 0.2
    w["l0.mix.dq"], w["l0.mix.dkv"] = dq, dkv
    uq, uk = w["l0.mix.uq"] * 0.05, w["l0.mix.uk"] * 0.05
    for h in range(heads):
        uq[h * (dim + rot_dim), 0] = 1.0
        uk[h * dim, 0] = 1.0
    w["l0.mix.uq"], w["l0.mix.uk"] = uq, uk
    return cfg, {n: bf16_bits(v) for n, v in w.items()}
