"""Virolorn on the GPU against the plain oracle (tests/virolorn_oracle.py): every mechanism, both activation precisions, and
every way of cutting a sequence into portions and steps."""
import numpy as np
import pytest

import virolorn_oracle as vo
from virolorn_util import FF, build, config, delta, far_key_model, latent, lightning, public, row_errors, tokens, values, weights

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 3e-5, 8e-2  # largest row error; bf16: the rows' root mean square stays below BF16_RMS
BF16_RMS = 3.5e-2

# one mechanism or size at a time; values that other models make equal or 1 differ here, and the other way round
CASES = {
    "lightning": config([lightning()]),
    "lightning one head": config([lightning(heads=1, dim=7, vdim=9)]),
    "lightning decays 0 and 1": config([lightning(heads=4, decay=[0.0, 1.0, 0.5, 0.999])]),
    "lightning wide values": config([lightning(heads=2, dim=8, vdim=70)]),
    "lightning wide keys": config([lightning(heads=2, dim=200, vdim=10)]),
    "lightning with feed-forward": config([lightning(mlp=FF)]),
    "delta": config([delta()]),
    "delta head for head": config([delta(heads=3, kv_heads=3, dim=16, vdim=16)]),
    "delta one q/k head": config([delta(heads=5, kv_heads=1, dim=33, vdim=7, ranks=(1, 3))]),
    "delta no convolution reach": config([delta(conv=1)]),
    "delta two taps": config([delta(conv=2)]),
    "delta three taps": config([delta(conv=3, dim=36)]),
    "delta long convolution": config([delta(conv=6)]),
    "delta odd sizes": config([delta(heads=6, kv_heads=3, dim=5, vdim=11, conv=3, ranks=(17, 5))], width=51),
    "delta wide keys": config([delta(heads=2, kv_heads=1, dim=200, vdim=40)]),
    "delta wider keys": config([delta(heads=2, kv_heads=2, dim=260, vdim=9)]),
    "delta wide low ranks": config([delta(ranks=(150, 3)), delta(dim=40, ranks=(5, 200))]),
    "delta wider low ranks": config([delta(heads=2, kv_heads=2, dim=256, vdim=9, ranks=(300, 140))]),
    "delta with feed-forward": config([delta(mlp=FF)]),
    "latent": config([latent()]),
    "latent one head": config([latent(heads=1, dim=6, rot_dim=2, vdim=5, kv_rank=9, q_rank=3)]),
    "latent many heads": config([latent(heads=20, dim=8, rot_dim=4, vdim=12, kv_rank=24, q_rank=16)]),
    "latent wide rotation": config([latent(dim=10, rot_dim=30, base=3.0)]),
    "latent small rotation base": config([latent(base=1.5)]),
    "latent odd sizes": config([latent(heads=5, dim=13, rot_dim=10, vdim=9, kv_rank=37, q_rank=29)], width=45),
    "latent with feed-forward": config([latent(mlp=FF)]),
    "feed-forward odd width": config([lightning(mlp={"kind": "dense", "ff": 27})]),
    "odd width": config([delta(), latent(), lightning(mlp=FF)], width=57, vocab=61),
    "residual factor 1": config([latent(), lightning()], mult=1.0),
    "weights used again": config([delta(mlp=FF), latent(), ("again", 0), ("again", 0), ("again", 1), lightning(), ("again", 5)]),
    "layers of different sizes": config([lightning(), delta(), lightning(heads=2, dim=9, vdim=30), latent(mlp=FF), delta(heads=2, kv_heads=1, dim=12, vdim=31, conv=2),
                                         latent(heads=2, dim=9, rot_dim=6, vdim=33, kv_rank=20, q_rank=11, mlp={"kind": "dense", "ff": 24})]),
}
_cache = {}


def check(got, want, tol):
    err = row_errors(got, want)
    assert err.max() < tol and (tol < 1e-3 or np.sqrt((err ** 2).mean()) < BF16_RMS), (err.max(), int(err.argmax()), np.sqrt((err ** 2).mean()))


def oracle(name, cfg, n, seed=0):
    key = (name, n, seed)
    if key not in _cache:
        w = weights(cfg)
        t = tokens(cfg, n, seed)
        _cache[key] = (w, t, *vo.forward(cfg, values(w), t))
    return _cache[key]


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
@pytest.mark.parametrize("name", CASES)
def test_mechanism(dev, name, dtype, tol):
    """A whole prompt, then the same tokens one by one through the decode step: logits everywhere, residual at the end."""
    cfg, n = CASES[name], 37
    w, t, logits, res = oracle(name, cfg, n)
    m = build(dev, cfg, w, n + 1, dtype=dtype)
    got = m.extend(t, range(n))
    check(got, logits, tol)
    check(m.read_hidden(n), res[-1], tol)
    m.release(0)
    one = []
    for tok in t:
        m.decode([tok], 1)
        one.append(m.read_logits())
    check(np.stack(one), logits, tol)
    check(m.read_hidden(1), res[-1][-1:], tol)
    assert m.seq_len() == n
    m.destroy()


MIXED = config([delta(mlp=FF), latent(mlp=FF), lightning(heads=2, dim=32, vdim=32, mlp=FF), delta(heads=2, kv_heads=1, dim=32, vdim=24, conv=3), ("again", 0),
                ("again", 1), ("again", 2)])


@pytest.mark.parametrize("max_rows", [0, 5])
@pytest.mark.parametrize("cuts", [[2] * 40, [1, 2, 3, 5, 7, 11, 13, 17, 21], [16, 16, 16, 32], [15, 2, 30, 2, 31], [79, 1], [3, 4, 64, 5, 4]])
def test_portions(dev, cuts, max_rows):
    """Whatever the portions (and the rows of a block inside them), every position has the same logits."""
    n = sum(cuts)
    w, t, logits, _ = oracle("mixed", MIXED, n)
    m = build(dev, MIXED, w, n, max_rows=max_rows)
    got, at = [], 0
    for c in cuts:
        got.append(m.extend(t[at:at + c], range(c)))
        at += c
    check(np.concatenate(got), logits, 2 * F32_TOL)
    m.destroy()


@pytest.mark.parametrize("dtype,tol", [("float32", 2 * F32_TOL), ("bfloat16", BF16_TOL)])
def test_steps_and_portions_mixed(dev, dtype, tol):
    """Decode steps and portions of one sequence in turn, also as its first token."""
    cuts = [1, 1, 4, 1, 20, 1, 1, 2, 1, 33, 1, 2, 1, 1]
    n = sum(cuts)
    w, t, logits, _ = oracle("mixed", MIXED, n)
    m = build(dev, MIXED, w, n, dtype=dtype)
    got, at = [], 0
    for c in cuts:
        if c == 1:
            m.decode([t[at]], 1)
            got.append(m.read_logits()[None])
        else:
            got.append(m.extend(t[at:at + c], range(c)))
        at += c
    check(np.concatenate(got), logits, tol)
    m.destroy()


def test_batch_of_unequal_sequences(dev):
    """Sequences decoded side by side (prompts of different lengths) equal each alone."""
    cfg, lens, steps = MIXED, [1, 2, 15, 40], 19
    w = weights(cfg)
    seqs = [tokens(cfg, n + steps, seed=i) for i, n in enumerate(lens)]
    refs = [vo.forward(cfg, values(w), s)[0] for s in seqs]
    for dtype, tol in (("float32", 2 * F32_TOL), ("bfloat16", BF16_TOL)):
        m = build(dev, cfg, w, 64, max_batch=len(lens), dtype=dtype)
        for i, n in enumerate(lens):
            got = m.extend(seqs[i][:n], range(n), seq=i)
            check(got, refs[i][:n], tol)
        for k in range(steps):
            m.decode([s[n + k] for s, n in zip(seqs, lens)], 1)
            got = m.read_logits(len(lens) * cfg["vocab"]).reshape(len(lens), -1)
            for i, n in enumerate(lens):
                assert row_errors(got[i], refs[i][n + k]) < tol
        m.destroy()


@pytest.mark.parametrize("dtype,tol", [("float32", 2 * F32_TOL), ("bfloat16", BF16_TOL)])
def test_slots_are_reused(dev, dtype, tol):
    """A freed slot's latents, recurrent state and histories do not reach the next sequence, short or long."""
    cfg = MIXED
    w = weights(cfg)
    m = build(dev, cfg, w, 64, max_batch=2, dtype=dtype)
    for seed, n in enumerate([50, 1, 3, 29, 2]):
        t = tokens(cfg, n, seed)
        ref = vo.forward(cfg, values(w), t)[0]
        for slot in (1, 0):
            m.release(slot)
            check(m.extend(t, range(n), seq=slot), ref, tol)
        m.release(0)
        for i in range(n):  # and through the decode step
            m.decode([t[i]], 1)
            assert row_errors(m.read_logits(cfg["vocab"]), ref[i]) < tol
    m.destroy()


def test_two_uses_of_a_layer_keep_their_own_state(dev):
    """Layers that share tensors: what one of them caches or accumulates is not the other's (the oracle has no sharing of
    state to get wrong; swapping the order of two such layers' states would show in every later token)."""
    cfg = config([delta(), ("again", 0), latent(), ("again", 2), lightning(), ("again", 4)])
    n = 30
    w, t, logits, _ = oracle("twice", cfg, n)
    m = build(dev, cfg, w, n)
    got = [m.extend(t[:9], range(9)), m.extend(t[9:11], range(2))]
    for i in range(11, n):
        m.decode([t[i]], 1)
        got.append(m.read_logits()[None])
    check(np.concatenate(got), logits, 2 * F32_TOL)
    bytes_once = build(dev, config([delta(), latent(), lightning()]), w2 := weights(config([delta(), latent(), lightning()])), n)
    assert m.state_bytes > 1.9 * bytes_once.state_bytes and m.weight_bytes == bytes_once.weight_bytes and w2
    bytes_once.destroy()
    m.destroy()


# ---- keys far away -----------------------------------------------------------------------------------
@pytest.mark.parametrize("sizes", [dict(), dict(heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=32), dict(heads=18, dim=32, rot_dim=16, vdim=32, kv_rank=272, q_rank=32)])
@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
def test_far_keys(dev, sizes, dtype, tol):
    """One key stands out and its value dominates the output of every later position: at the sequence's start, at borders of
    the kernels' key tiles, just behind a portion's start, and for queries hundreds of tokens on, in prompts, portions and
    decoding."""
    cfg, w = far_key_model(**sizes)
    v, n, tail = values(w), 300, 10
    for place in (0, 31, 32, 63, 64, 127, 160, 200, 289):
        t = 2 + tokens(cfg, n, 4) % 38
        t[place] = 1
        ref = vo.forward(cfg, v, t)[0]
        m = build(dev, cfg, w, n, dtype=dtype)
        check(m.extend(t, range(n)), ref, tol)
        m.release(0)
        got, at = [], 0
        for c in (place + 1, 2, 50, n):
            c = min(c, n - tail - at)
            if c > 0:
                got.append(m.extend(t[at:at + c], range(c)))
                at += c
        for i in range(at, n):
            m.decode([t[i]], 1)
            got.append(m.read_logits()[None])
        check(np.concatenate(got), ref, tol)
        m.destroy()


def test_tokens_after_a_position_do_not_reach_it(dev):
    cfg, n = MIXED, 40
    w = weights(cfg)
    a, b = tokens(cfg, n, 1), tokens(cfg, n, 2)
    b[:23] = a[:23]
    for dtype in ("float32", "bfloat16"):
        m = build(dev, cfg, w, n, dtype=dtype)
        x = m.extend(a, range(n))
        m.release(0)
        y = m.extend(b, range(n))
        m.destroy()
        assert np.array_equal(x[:23], y[:23]) and row_errors(x[23:], y[23:]).min() > 0.1


# ---- recurrences with a long memory --------------------------------------------------------------------
def test_a_far_write_is_still_there(dev):
    """Decays of 1 or close to it: what the first tokens wrote reaches the last ones, and it is the writes that differ."""
    cfg = config([lightning(heads=2, dim=16, vdim=16, decay=[1.0, 0.9999]), delta(heads=2, kv_heads=1, dim=16, vdim=16)], mult=1.0)
    w = values(weights(cfg, 5))
    w["l1.mix.A_log"] = np.full(2, -9.0)
    w["l1.mix.dt_bias"] = np.full(32, -6.0)
    w["l1.mix.b"] *= 0.2
    from doppler_b200.safetensors import bf16_bits
    bits = {k: bf16_bits(x) for k, x in w.items()}
    n = 260
    t = tokens(cfg, n, 3)
    u = t.copy()
    u[:2] = (t[:2] + 1) % cfg["vocab"]
    ref, other = vo.forward(cfg, values(bits), t)[0], vo.forward(cfg, values(bits), u)[0]
    assert row_errors(other[-20:], ref[-20:]).min() > 50 * F32_TOL
    m = build(dev, cfg, bits, n)
    got = [m.extend(t[:255], range(255))]
    for i in range(255, n):
        m.decode([t[i]], 1)
        got.append(m.read_logits()[None])
    check(np.concatenate(got), ref, 4 * F32_TOL)
    m.destroy()


def test_strong_decays(dev):
    """Decays down to nothing: channels that forget at once beside channels that keep everything."""
    cfg = config([delta(heads=2, kv_heads=2, dim=32, vdim=16), lightning(heads=3, dim=32, vdim=16, decay=[0.0, 1e-12, 1.0])])
    w = values(weights(cfg, 6))
    w["l0.mix.A_log"] = np.array([3.5, 2.0])
    w["l0.mix.dt_bias"] = np.where(np.arange(64) % 3 == 0, 12.0, np.where(np.arange(64) % 3 == 1, -9.0, 0.5))
    from doppler_b200.safetensors import bf16_bits
    bits = {k: bf16_bits(x) for k, x in w.items()}
    n = 150
    t = tokens(cfg, n, 3)
    ref = vo.forward(cfg, values(bits), t)[0]
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
        m = build(dev, cfg, bits, n, dtype=dtype)
        check(m.extend(t, range(n)), ref, tol)
        m.destroy()


def test_long_decoding(dev):
    """Several hundred decode steps: recurrent state, the convolutions' rings, and the split of the keys."""
    cfg = config([delta(dim=24), latent(), lightning(), delta(conv=2)])
    n, pre = 420, 3
    w, t, logits, _ = oracle("long", cfg, n)
    for dtype, tol in (("float32", 4 * F32_TOL), ("bfloat16", BF16_TOL)):
        m = build(dev, cfg, w, n, dtype=dtype)
        m.extend(t[:pre])
        errs = []
        for i in range(pre, n):
            m.decode([t[i]], 1)
            errs.append(row_errors(m.read_logits(), logits[i]))
        assert max(errs) < tol
        m.destroy()


# ---- the kernels of the larger sizes (bf16) --------------------------------------------------------
LARGE = {
    "delta 128": config([delta(heads=8, kv_heads=4, dim=128, vdim=64, ranks=(64, 32))], width=128),
    "delta 64": config([delta(heads=4, kv_heads=4, dim=64, vdim=128, conv=3, ranks=(40, 24))], width=128),
    "delta 32": config([delta(heads=6, kv_heads=2, dim=32, vdim=40, conv=2, ranks=(16, 16))], width=128),
    "delta 256": config([delta(heads=2, kv_heads=1, dim=256, vdim=48, ranks=(128, 8))], width=128),
    "lightning 128 x 16": config([lightning(heads=4, dim=128, vdim=16)], width=128),
    "lightning 64 x 32": config([lightning(heads=96, dim=64, vdim=32)], width=128),
    "lightning 32 x 64": config([lightning(heads=90, dim=32, vdim=64)], width=128),
    "lightning 128 x 64": config([lightning(heads=90, dim=128, vdim=64)], width=128),
    # expanded keys (three sizes of the prompt kernel) and the absorbed decode kernel (two)
    "latent 64": config([latent(heads=4, dim=40, rot_dim=16, vdim=56, kv_rank=96, q_rank=64)], width=128),
    "latent 64, sizes padded": config([latent(heads=3, dim=21, rot_dim=10, vdim=27, kv_rank=50, q_rank=40)], width=128),
    "latent 128": config([latent(heads=6, dim=64, rot_dim=32, vdim=72, kv_rank=160, q_rank=96)], width=128),
    "latent 192": config([latent(heads=8, dim=128, rot_dim=64, vdim=128, kv_rank=512, q_rank=192, scale=0.07)], width=128),
    "latent 192, sizes padded": config([latent(heads=2, dim=101, rot_dim=38, vdim=77, kv_rank=300, q_rank=72, scale=0.09)], width=128),
    # beyond both: absorbed prompts, the generic kernel
    "latent wide values": config([latent(heads=3, dim=32, rot_dim=16, vdim=160, kv_rank=64, q_rank=64)], width=128),
    "latent wide": config([latent(heads=2, dim=64, rot_dim=32, vdim=48, kv_rank=600, q_rank=64, scale=0.1)], width=128),
    "wide": config([latent(mlp={"kind": "dense", "ff": 700}), lightning(mlp={"kind": "dense", "ff": 500})], width=264, vocab=600),
}


@pytest.mark.parametrize("name", LARGE)
def test_large_sizes_bf16(dev, name):
    """Prompts and portions around the recurrences' chunks and the tiles of products and attention, then decoding."""
    cfg, n, tail = LARGE[name], 333, 6
    w, t, logits, _ = oracle(name, cfg, n)
    m = build(dev, cfg, w, n, dtype="bfloat16")
    for cuts in ([n - tail], [63, 65, 2, 64, 17, n - tail - 211], [200, 1, n - tail - 201]):
        m.release(0)
        got, at = [], 0
        for c in cuts:
            got.append(m.extend(t[at:at + c], range(c)))
            at += c
        for i in range(at, n):
            m.decode([t[i]], 1)
            got.append(m.read_logits()[None])
        check(np.concatenate(got), logits, BF16_TOL / 2)
    m.destroy()


def test_many_keys_split_over_ctas_bf16(dev):
    """A sequence so long that decoding and short portions split its keys, in the second slot too."""
    cfg = config([latent(heads=18, dim=64, rot_dim=32, vdim=64, kv_rank=128, q_rank=64, scale=0.2)], width=128)
    n = 700
    w, t, logits, _ = oracle("many keys", cfg, n)
    m = build(dev, cfg, w, 2100, max_batch=2, dtype="bfloat16")
    got = [m.extend(t[:660], range(640, 660)), m.extend(t[660:667], range(7))]
    for i in range(667, n):
        m.decode([t[i]], 1)
        got.append(m.read_logits(cfg["vocab"])[None])
    check(np.concatenate(got), logits[640:], BF16_TOL / 2)
    got = [m.extend(t[:660], range(640, 660), seq=1), m.extend(t[660:], range(40), seq=1)]
    check(np.concatenate(got), logits[640:], BF16_TOL / 2)
    m.destroy()


def test_recurrences_are_32_bit(dev):
    """What bf16 changes are the operands of the projections; the recurrences themselves agree with the 32-bit mode closely
    where those are exact: embeddings of +-1, one-hot projections, convolutions and gates that pass them on."""
    W, H, D, V = 64, 2, 32, 16
    rng = np.random.default_rng(8)
    cfg = config([delta(heads=H, kv_heads=H, dim=D, vdim=V, conv=1, ranks=(8, 8))], width=W, vocab=50, eps=1e-5, mult=1.0)
    w = values(weights(cfg, 8))
    w["embed"] = np.where(rng.random((50, W)) < 0.5, 1.0, -1.0)
    w["l0.norm1"] = np.ones(W)

    def pick(n):
        p = np.zeros((n, W))
        p[np.arange(n), rng.integers(0, W, n)] = 1.0
        return p

    for name, n in (("q", H * D), ("k", H * D), ("v", H * V)):
        w["l0.mix." + name] = pick(n)
        w[f"l0.mix.{name}.conv"] = np.full((n, 1), 1.0)
    w["l0.mix.a1"], w["l0.mix.g1"] = pick(8), pick(8)
    w["l0.mix.g2"] = np.zeros((H * V, 8))
    from doppler_b200.safetensors import bf16_bits
    bits = {k: bf16_bits(x) for k, x in w.items()}
    n = 300
    t = tokens(cfg, n, 2)
    _, res = vo.forward(cfg, values(bits), t)
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", 4e-3)):
        m = build(dev, cfg, bits, n, dtype=dtype)
        m.extend(t)
        assert row_errors(m.read_hidden(n), res[-1]).max() < tol  # in bf16: the output projection's operand is left
        m.destroy()


# ---- generation -------------------------------------------------------------------------------------
def _greedy(cfg, v, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(vo.forward(cfg, v, out)[0][-1].argmax()))
    return out[len(prompt):]


def _generation_model():
    """Small embeddings: what the layers add decides the next token, not the token itself."""
    from doppler_b200.safetensors import bf16_bits

    cfg = dict(MIXED, norm={"eps": 1e-6})
    w = weights(cfg, 22)
    w["embed"] = bf16_bits(0.1 * values(w)["embed"])
    return cfg, w


def _write_model(path, cfg, w):
    import json

    from doppler_b200.safetensors import write_bf16

    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(public(cfg)))
    write_bf16(str(path / "model.safetensors"), w)


@pytest.mark.parametrize("batch", [1, 3])
def test_greedy_generation(dev, tmp_path, batch):
    """Through the registry, the weight loading and the scheduler, from a model folder; prompts of different lengths, more of
    them than slots."""
    from doppler_b200.registry import load_model
    from doppler_b200.scheduler import Scheduler

    cfg, w = _generation_model()
    _write_model(tmp_path / "model", cfg, w)
    prompts = [tokens(cfg, n, 30 + n).tolist() for n in (5, 1, 18, 33)]
    m = load_model(dev, str(tmp_path / "model"), 64, batch, "float32")
    got = Scheduler(m).generate(prompts, 24, block=7)
    stop = got[0][10]
    stopped = Scheduler(m).generate(prompts[:1], 24, stop=[stop])
    m.destroy()
    for p, toks in zip(prompts, got):
        assert toks == _greedy(cfg, values(w), p, 24)
    assert stopped[0] == got[0][:got[0].index(stop) + 1]
    assert len(set(sum(got, []))) > 10, "decoding collapsed; the comparison would be vacuous"


def test_command_line_and_trace(dev, tmp_path):
    """`python -m doppler_b200 generate` and bin/trace_run, as a user starts them."""
    import json
    import os
    import subprocess
    import sys

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg, w = _generation_model()
    model = tmp_path / "model"
    _write_model(model, cfg, w)
    prompt = tokens(cfg, 9, 3).tolist()
    res = subprocess.run([sys.executable, "-m", "doppler_b200", "generate", "--model", str(model), "--prompt", ",".join(map(str, prompt)), "--max-new", "12",
                          "--dtype", "float32"], cwd=root, capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr
    assert json.loads(res.stdout.splitlines()[-1])["tokens"] == _greedy(cfg, values(w), prompt, 12)
    w = weights(cfg, 23)
    _write_model(model, cfg, w)
    t = tokens(cfg, 40, 4).tolist()
    ref = vo.forward(cfg, values(w), t)[0]
    short = tokens(cfg, 3, 5).tolist()
    ref2 = vo.forward(cfg, values(w), short)[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:30], "want": [0, 29, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[30:31], "want": [0]}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": t[31:], "want": [8]}], "end": ["a"]},
             {"step": 3, "entries": [{"id": "b", "tokens": short, "want": [0, 1, 2]}], "end": ["b"]}]
    for dtype, tol in (("float32", 2 * F32_TOL), ("bfloat16", BF16_TOL)):
        out = tmp_path / dtype
        out.mkdir()
        res = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", dtype, "--out", str(out), "--max-tokens", "40"],
                             input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
        assert res.returncode == 0, res.stderr
        assert [x for x in res.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
        for i, want in enumerate((ref[[0, 29, 7]], ref[[30]], ref[[39]], ref2)):
            check(np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"]), want, tol)


def test_bad_descriptions_and_weights_are_refused(dev):
    from doppler_b200 import _lib as L
    from doppler_b200 import virolorn
    from doppler_b200.model import StackModel

    cfg = config([lightning(), delta(), ("again", 1), latent()])
    w = weights(cfg)
    stack, layers = virolorn.stack_config(public(cfg), lambda n: w[n].shape if n in w else None)
    m = StackModel(dev, stack, layers, 16)
    with pytest.raises(Exception, match="has not been loaded"):
        m.prefill([1, 2, 3])
    with pytest.raises(Exception, match="expects shape"):
        m.load_tensor(1, L.T_A2, w["l1.mix.a2"][:, :-1].copy())
    with pytest.raises(Exception, match="has no"):
        m.load_tensor(0, L.T_UQ, w["l3.mix.uq"])
    with pytest.raises(Exception, match="uses the tensors of layer 1"):
        m.load_tensor(2, L.T_Q, w["l1.mix.q"])
    m.destroy()
    for change, text in ((dict(share=1), "cannot use"), (dict(kv_heads=3, share=0), "heads over"), (dict(vdim=13), "cannot use")):
        bad = [dict(l) for l in layers]
        bad[2].update(change)
        with pytest.raises(Exception, match=text):
            StackModel(dev, stack, bad, 16)
    with pytest.raises(Exception, match="norms behind"):
        StackModel(dev, dict(stack, post_norm=0), layers, 16)
