"""Virolorn without a GPU: the oracle against restatements of its recurrences, that the test weights make mistakes visible,
configuration, registry and command line."""
import copy
import json

import numpy as np
import pytest

import virolorn_oracle as vo
from doppler_b200 import _lib as L
from doppler_b200 import registry, virolorn
from doppler_b200.safetensors import write_bf16
from virolorn_util import FF, config, delta, far_key_model, latent, lightning, public, row_errors, tokens, values, weights

CFG = config([delta(mlp=FF), latent(mlp=FF), lightning(mlp=FF), delta(heads=3, kv_heads=3, dim=8, vdim=24, conv=2), ("again", 0), ("again", 1), ("again", 2)])
BF16_TOL, BF16_RMS = 8e-2, 3.5e-2  # the loosest tolerances of the GPU tests (largest row error, root mean square of the rows)


def shape_of(w):
    return lambda n: w[n].shape if n in w else None


# ---- oracle -----------------------------------------------------------------------------------------
def test_constant_decay_recurrence_equals_its_sum():
    rng = np.random.default_rng(0)
    T, H, D, V = 8, 3, 4, 5
    q, k, v, decay = rng.standard_normal((T, H, D)), rng.standard_normal((T, H, D)), rng.standard_normal((T, H, V)), np.array([0.3, 0.9, 1.0])
    o = vo.decayed_sum_scan(q, k, v, decay)
    for t in range(T):
        for h in range(H):
            assert np.allclose(o[t, h], sum(decay[h] ** (t - s) * (q[t, h] @ k[s, h]) * v[s, h] for s in range(t + 1)))


def test_delta_recurrence_equals_its_matrix_form():
    """S_t = (I - beta k k^T) diag(g) S_(t-1) + beta k v^T"""
    rng = np.random.default_rng(1)
    T, H, D, V = 9, 2, 4, 3
    q, k, v = rng.standard_normal((T, H, D)), rng.standard_normal((T, H, D)), rng.standard_normal((T, H, V))
    g, beta = rng.uniform(0.2, 1, (T, H, D)), rng.uniform(0, 1, (T, H))
    o = vo.delta_scan(q, k, v, g, beta)
    for h in range(H):
        S = np.zeros((D, V))
        for t in range(T):
            kk = k[t, h][:, None]
            S = (np.eye(D) - beta[t, h] * kk @ kk.T) @ (g[t, h][:, None] * S) + beta[t, h] * kk @ v[t, h][None]
            assert np.allclose(o[t, h], S.T @ q[t, h])


def test_rotation_is_relative():
    rng = np.random.default_rng(2)
    a, b = rng.standard_normal(6), rng.standard_normal(6)
    x = vo.rotate_half(np.repeat(a[None], 30, 0), 20.0)
    y = vo.rotate_half(np.repeat(b[None], 30, 0), 20.0)
    assert np.allclose(x[0], a) and np.isclose(x[9] @ y[4], x[25] @ y[20]) and not np.isclose(x[9] @ y[4], x[9] @ y[5])


def test_oracle_is_causal_and_prefix_consistent():
    w, t = values(weights(CFG)), tokens(CFG, 30)
    whole = vo.forward(CFG, w, t)[0]
    for n in (1, 2, 17):
        assert np.allclose(vo.forward(CFG, w, t[:n])[0], whole[:n])


def _mistakes():
    def mixer(i, **kw):
        return lambda c, w: c["layers"][i]["mixer"].update(kw)

    yield "score scale", mixer(1, scale=0.2)
    yield "rotation base", mixer(1, rot={"base": 500.0, "dims": 8})
    yield "decays in another order", lambda c, w: c["layers"][2]["mixer"]["decay"].reverse()
    yield "residual factor left out", lambda c, w: c.update(residual_mult=1.0)

    def zero(*names):
        def plant(c, w):
            for n in names:
                w[n] = np.zeros_like(w[n])
        return plant

    for name in ("l0.mix.q.conv", "l0.mix.b", "l0.mix.a2", "l0.mix.g2", "l0.mix.dt_bias", "l0.mix.A_log", "l1.mix.g", "l2.mix.g", "l1.mix.uk"):
        yield "without " + name, zero(name)
    yield "without the rotated part", lambda c, w: w.update({"l1.mix.dkv": np.concatenate([w["l1.mix.dkv"][:40], np.zeros((8, 64))])})

    def ones(name):
        return lambda c, w: w.update({name: np.ones_like(w[name])})

    for name in ("l0.norm1b", "l1.norm2b", "l0.mix.norm", "l1.mix.dq.norm", "l1.mix.dkv.norm", "l2.mix.norm"):
        yield "weight of " + name, ones(name)

    def reverse(name):
        return lambda c, w: w.update({name: w[name][:, ::-1].copy()})

    yield "taps reversed", reverse("l0.mix.v.conv")

    def dims(c, w):  # rotated part first instead of last in every head's query
        a = w["l1.mix.uq"].reshape(3, 32, -1)
        w["l1.mix.uq"] = np.concatenate([a[:, 24:], a[:, :24]], 1).reshape(96, -1)

    yield "parts of the query swapped", dims

    def interleave(c, w):  # rotation of neighbouring dimensions instead of halves
        perm = [0, 4, 1, 5, 2, 6, 3, 7]
        a = w["l1.mix.dkv"].copy()
        a[40:] = a[40:][perm]
        w["l1.mix.dkv"] = a

    yield "other rotation pairs", interleave

    def kv_heads(c, w):  # heads dealt to the q/k heads in turn instead of in runs
        d = w["l0.mix.v"].reshape(4, 12, -1)[[0, 2, 1, 3]].reshape(48, -1)
        w["l0.mix.v"] = d

    yield "heads dealt in turn", kv_heads


@pytest.mark.parametrize("name,plant", list(_mistakes()), ids=[n for n, _ in _mistakes()])
def test_mistakes_show(name, plant):
    """Every planted mistake moves some position's logits by more than the tolerances of the GPU tests."""
    w, t = values(weights(CFG)), tokens(CFG, 40)
    good = vo.forward(CFG, w, t)[0]
    cfg, bad = copy.deepcopy(CFG), dict(w)
    plant(cfg, bad)
    err = row_errors(vo.forward(cfg, bad, t)[0], good)
    assert err.max() > 2 * BF16_TOL or np.sqrt((err ** 2).mean()) > 1.3 * BF16_RMS


def test_a_far_key_shows():
    """In the far-key model every position's logits depend on the one key that stands out, however far back it is."""
    cfg, w = far_key_model()
    v = values(w)
    t = 2 + tokens(cfg, 200, 4) % 38
    u = t.copy()
    u[3] = 1
    err = row_errors(vo.forward(cfg, v, u)[0], vo.forward(cfg, v, t)[0])
    assert err[:3].max() < 1e-12 and err[4:].min() > 0.16


# ---- configuration -------------------------------------------------------------------------------------
def test_stack_config_takes_everything_from_the_configuration_and_the_shapes():
    w = weights(CFG)
    stack, layers = virolorn.stack_config(public(CFG), shape_of(w))
    assert stack == {"width": 64, "vocab": 97, "streams": 1, "norm_groups": 1, "input_taps": 0, "eps": 1e-4, "embed_scale": 1.0, "post_norm": 1, "residual_mult": 0.7}
    ff = {"ff": 40, "ff_limit": 0.0, "ff_slope": 1.0, "ff_shift": 0.0}
    assert layers[0] == {"heads": 4, "vdim": 12, "mixer": L.MIXER_DELTA, "kv_heads": 2, "dim": 20, "conv_taps": 4, "decay_rank": 6, "gate_rank": 10, **ff}
    assert layers[1] == {"heads": 3, "vdim": 20, "mixer": L.MIXER_LATENT, "dim": 24, "rot_dim": 8, "kv_rank": 40, "q_rank": 24, "scale": 0.35, "rot_base": 50.0,
                         "head_gate": 1, **ff}
    assert layers[2]["mixer"] == L.MIXER_LIGHTNING and layers[2]["decay"] == CFG["layers"][2]["mixer"]["decay"]
    assert "ff" not in layers[3] and layers[3]["decay_rank"] == 6
    assert [l.get("share", 0) for l in layers] == [0, 0, 0, 0, 1, 2, 3] and layers[4]["gate_rank"] == 10
    assert {n for n, _, _ in virolorn.model_tensors(layers)} == set(w)


def test_weights_of_a_layer_that_borrows_itself():
    cfg = public(config([lightning(), ("again", 0), ("again", 1)]))
    assert [l.get("share", 0) for l in virolorn.stack_config(cfg, lambda n: None)[1]] == [0, 1, 1]


@pytest.mark.parametrize("change,text", [
    (lambda c: c.update(architecture="Other"), "is not Virolorn"),
    (lambda c: c.pop("residual_mult"), "missing residual_mult"),
    (lambda c: c["layers"][0].update(type="rwkv"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "missing scale"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=6), "rotated dimensions"),
    (lambda c: c["layers"][2]["mixer"]["decay"].pop(), "decays for"),
    (lambda c: c["layers"][2]["mixer"]["decay"].__setitem__(0, 1.5), "between 0 and 1"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: c["layers"][1]["mixer"].update(kv_rank=0), "not a positive number"),
    (lambda c: c["layers"][4].update(weights_of=4), "does not lead"),
    (lambda c: c["layers"][4].update(weights_of=9), "does not lead"),
    (lambda c: c["layers"][4].update(weights_of=2), "differs from it"),
])
def test_bad_configurations_are_named(change, text):
    c = copy.deepcopy(public(CFG))
    change(c)
    with pytest.raises(virolorn.ConfigError, match=text):
        virolorn.stack_config(c, shape_of(weights(CFG)))


def test_sizes_that_only_a_tensor_has():
    with pytest.raises(virolorn.ConfigError, match="l0.mix.a1"):
        virolorn.stack_config(public(CFG), lambda n: None)


def test_registry_and_info(tmp_path, capsys):
    from doppler_b200 import __main__ as cli

    (tmp_path / "config.json").write_text(json.dumps(public(CFG)))
    write_bf16(str(tmp_path / "model.safetensors"), weights(CFG))
    assert registry.describe(str(tmp_path))["kind"] == "Virolorn"
    assert cli.info(["--model", str(tmp_path)]) == 0
    d = json.loads(capsys.readouterr().out)
    assert d["kind"] == "Virolorn" and len(d["layers"]) == 7 and d["layers"][0]["decay_rank"] == 6
