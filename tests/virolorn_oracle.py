"""Plain, slow restatement of the Virolorn decoder's mechanisms, one function per equation.

numpy in float64, one sequence at a time, no cache: every function sees the whole sequence and walks it token by token
where the mechanism is a recurrence.  It shares no code with the product path (weights arrive as plain arrays, the
configuration as the dictionary of config.json).
"""
import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms_norm(x, w, eps):
    """over the last axis"""
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def short_conv(x, w):
    """x [T, C], w [C, taps]: the last column multiplies the row itself, the first the row taps - 1 before; then silu."""
    T, C = x.shape
    taps = w.shape[1]
    y = np.zeros((T, C))
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                y[t] += w[:, j] * x[s]
    return silu(y)


def unit(x):
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def decayed_sum_scan(q, k, v, decay):
    """q, k [T, H, D], v [T, H, V], decay [H]: S = decay S + k v^T, o = S^T q."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def lightning(h, m, w, eps):
    T = h.shape[0]
    H, D, V = m["heads"], m["dim"], m["vdim"]
    q = silu(h @ w["q"].T).reshape(T, H, D)
    k = silu(h @ w["k"].T).reshape(T, H, D)
    v = silu(h @ w["v"].T).reshape(T, H, V)
    o = decayed_sum_scan(q, k, v, np.asarray(m["decay"], np.float64)).reshape(T, H * V)
    return (rms_norm(o, w["norm"], eps) * sigmoid(h @ w["g"].T)) @ w["o"].T


def delta_scan(q, k, v, g, beta):
    """q, k, g [T, H, D], v [T, H, V], beta [T, H]: S = g S (per key channel), u = beta (v - S^T k), S += k u^T, o = S^T q."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2]))
    o = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = g[t][:, :, None] * S
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        o[t] = np.einsum("hdv,hd->hv", S, q[t])
    return o


def channel_decay(h, w, H, D):
    T = h.shape[0]
    a = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
    return np.exp(-np.exp(w["A_log"])[None, :, None] * softplus(a).reshape(T, H, D))


def channel_delta(h, m, w, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w["q"].T, w["q.conv"]).reshape(T, G, D)
    k = short_conv(h @ w["k"].T, w["k.conv"]).reshape(T, G, D)
    v = short_conv(h @ w["v"].T, w["v.conv"]).reshape(T, H, V)
    of = np.arange(H) // (H // G)
    q, k = unit(q)[:, of] / np.sqrt(D), unit(k)[:, of]
    o = delta_scan(q, k, v, channel_decay(h, w, H, D), sigmoid(h @ w["b"].T))
    o = rms_norm(o, w["norm"], eps).reshape(T, H * V) * sigmoid((h @ w["g1"].T) @ w["g2"].T)
    return o @ w["o"].T


def rotate_half(x, base):
    """x [T, ..., R], row t at position t: dimension i with dimension i + R / 2."""
    T, R = x.shape[0], x.shape[-1]
    f = base ** (-2.0 * np.arange(R // 2) / R)
    a = (np.arange(T)[:, None] * f).reshape((T,) + (1,) * (x.ndim - 2) + (R // 2,))
    u, v = x[..., :R // 2], x[..., R // 2:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)], axis=-1)


def causal_softmax(s):
    """s [T, T], row = query"""
    T = s.shape[0]
    s = np.where(np.arange(T)[None, :] <= np.arange(T)[:, None], s, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    return e / e.sum(axis=1, keepdims=True)


def latent_attention(h, m, w, eps):
    T = h.shape[0]
    H, D, R, V, K = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(T, H, D + R)
    down = h @ w["dkv"].T
    c = rms_norm(down[:, :K], w["dkv.norm"], eps)
    k_rot = rotate_half(down[:, K:], m["rot"]["base"])
    q_rot = rotate_half(q[:, :, D:], m["rot"]["base"])
    k = (c @ w["uk"].T).reshape(T, H, D)
    v = (c @ w["uv"].T).reshape(T, H, V)
    gate = sigmoid(h @ w["g"].T)
    o = np.zeros((T, H, V))
    for hh in range(H):
        o[:, hh] = causal_softmax((q[:, hh, :D] @ k[:, hh].T + q_rot[:, hh] @ k_rot.T) * m["scale"]) @ v[:, hh]
    return (o * gate[:, :, None]).reshape(T, H * V) @ w["o"].T


def gated_ff(h, w):
    return (silu(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


MIXERS = {"lightning": lightning, "channel_delta": channel_delta, "latent_attention": latent_attention}


def sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(cfg, w, tokens):
    """Returns (logits [T, vocab], residual [layers, T, width])."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w["embed"][np.asarray(tokens)]
    res = []
    for i, layer in enumerate(cfg["layers"]):
        src = i
        while "weights_of" in cfg["layers"][src]:
            src = cfg["layers"][src]["weights_of"]
        lw = sub(w, f"l{src}.")
        y = MIXERS[layer["type"]](rms_norm(x, lw["norm1"], eps), layer["mixer"], sub(lw, "mix."), eps)
        x = x + mult * rms_norm(y, lw["norm1b"], eps)
        if layer["mlp"] is not None:
            y = gated_ff(rms_norm(x, lw["norm2"], eps), sub(lw, "mlp."))
            x = x + mult * rms_norm(y, lw["norm2b"], eps)
        res.append(x)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T, np.stack(res)
