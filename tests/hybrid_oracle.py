"""Plain, slow restatement of the hybrid decoder's mechanisms (Fenorax), one function per equation.

numpy in float64, one sequence at a time, no cache: every function sees the whole sequence.  It shares no
code with the product path (weights arrive as plain arrays, the configuration as the dictionary of
config.json).
"""
import numpy as np


def silu(z):
    return z / (1.0 + np.exp(-z))


def softplus(z):
    return np.logaddexp(0.0, z)


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def grouped_rms_norm(x, w, groups, eps):
    """x [T, C]: every one of the `groups` equal parts by its own root mean square, then times w."""
    T, C = x.shape
    p = x.reshape(T, groups, C // groups)
    p = p / np.sqrt(np.mean(p * p, axis=-1, keepdims=True) + eps)
    return p.reshape(T, C) * w


def causal_conv(x, w, b=None):
    """x [T, C], w [C, taps]: w[:, taps - 1] multiplies the row itself, w[:, 0] the row taps - 1 before; rows before 0 count as 0."""
    T, C = x.shape
    taps = w.shape[1]
    pad = np.concatenate([np.zeros((taps - 1, C)), x])
    y = np.zeros((T, C))
    for j in range(taps):
        y += pad[j:j + T] * w[:, j]
    return y if b is None else y + b


def input_conv(h, w):
    return h + causal_conv(h, w)


def stream_read(xs, w_in):
    """xs [streams, T, C] -> u [T, C]"""
    return np.einsum("s,stc->tc", w_in, xs)


def stream_write(xs, mix, w_out, y):
    """mix is indexed [from, to]"""
    return np.einsum("st,snc->tnc", mix, xs) + w_out[:, None, None] * y[None]


def ssd_scan(x, B, C, dt, A_log, D):
    """x [T, heads, P], B and C [T, groups, N], dt [T, heads] (after softplus) -> y [T, heads, P]"""
    T, H, P = x.shape
    G, N = B.shape[1:]
    S = np.zeros((H, N, P))
    y = np.zeros((T, H, P))
    g = np.arange(H) // (H // G)
    for t in range(T):
        decay = np.exp(-np.exp(A_log) * dt[t])
        S = decay[:, None, None] * S + dt[t][:, None, None] * B[t][g][:, :, None] * x[t][:, None, :]
        y[t] = np.einsum("hnp,hn->hp", S, C[t][g]) + D[:, None] * x[t]
    return y


def mamba2(h, m, w, eps):
    """h [T, C]; m: the mixer's sizes; w: name -> array (in, conv, conv.b, dt_bias, A_log, D, norm, o)"""
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    p = h @ w["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, w["conv"], w["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, P)
    B = xbc[:, inner:inner + G * N].reshape(T, G, N)
    C = xbc[:, inner + G * N:].reshape(T, G, N)
    y = ssd_scan(x, B, C, softplus(dt + w["dt_bias"]), w["A_log"], w["D"]).reshape(T, inner)
    y = grouped_rms_norm(y * silu(z), w["norm"], m["norm_groups"], eps)
    return y @ w["o"].T


def chunk_attention(q, k, v, scale, chunk):
    """q [T, H, D], k [T, G, D], v [T, G, V]: causal, and both positions in the same chunk"""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    see = (j <= i) & (i // chunk == j // chunk)
    for hh in range(H):
        g = hh // (H // G)
        s = np.where(see, (q[:, hh] @ k[:, g].T) * scale, -np.inf)
        s = np.exp(s - s.max(axis=1, keepdims=True))
        out[:, hh] = (s / s.sum(axis=1, keepdims=True)) @ v[:, g]
    return out


def unit_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def attention(h, m, w, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit_rms((h @ w["q"].T).reshape(T, H, D), eps)
    k = unit_rms((h @ w["k"].T).reshape(T, G, D), eps)
    v = (h @ w["v"].T).reshape(T, G, V)
    o = chunk_attention(q, k, v, m["scale"], m["mask"]["size"])
    o = o * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * V) @ w["o"].T


def clamped_glu(h, limit, w):
    g = np.minimum(h @ w["gate"].T, limit)
    u = np.clip(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ w["down"].T


MIXERS = {"mamba2": mamba2, "attention": attention}


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg, w, tokens):
    """Returns (logits [T, vocab], residual [layers, T, width]: the sum of the streams after every layer)."""
    eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    xs = np.repeat(x[None], cfg["streams"], axis=0)
    res = []
    for i, layer in enumerate(cfg["layers"]):
        lw = sub(w, f"l{i}.")
        for q, block in (("1", lambda h: MIXERS[layer["type"]](h, layer["mixer"], sub(lw, "mix."), eps)),
                         ("2", lambda h: clamped_glu(h, layer["mlp"]["limit"], sub(lw, "mlp.")))):
            if q == "2" and layer["mlp"] is None:
                continue
            h = grouped_rms_norm(stream_read(xs, lw[f"hc{q}.in"]), lw[f"norm{q}"], groups, eps)
            xs = stream_write(xs, lw[f"hc{q}.mix"], lw[f"hc{q}.out"], block(input_conv(h, lw[f"canon{q}"])))
        res.append(xs.sum(axis=0))
    return grouped_rms_norm(xs.sum(axis=0), w["final.norm"], groups, eps) @ w["embed"].T, np.stack(res)
