"""Fenorax on the GPU against the plain oracle (tests/hybrid_oracle.py): every mechanism, both activation precisions, and
every way of cutting a sequence into portions and steps."""
import numpy as np
import pytest

import hybrid_oracle as ho
from fenorax_util import attention, build, config, mamba, row_errors, tokens, values, weights

pytestmark = pytest.mark.gpu

F32_TOL, BF16_TOL = 3e-5, 8e-2  # largest row error; bf16: the rows' root mean square stays below BF16_RMS
BF16_RMS = 3.5e-2
GLU = {"kind": "dense", "ff": 40, "limit": 0.75}

# one mechanism or size at a time; values that other models make equal or 1 differ here, and the other way round
CASES = {
    "mamba": config([mamba()]),
    "mamba one group": config([mamba(heads=3, groups=1, norm_groups=1)]),
    "mamba group per head": config([mamba(heads=4, groups=4, norm_groups=4)]),
    "mamba norm groups other than groups": config([mamba(heads=6, groups=2, norm_groups=3)]),
    "mamba odd sizes": config([mamba(heads=3, vdim=7, state=5, groups=3, conv=3, norm_groups=7)], width=30, groups=5),
    "mamba wide state": config([mamba(heads=2, vdim=33, state=200, groups=1, norm_groups=2)]),
    "mamba no convolution reach": config([mamba(conv=1)]),
    "mamba long convolution": config([mamba(conv=7)]),
    "mamba with feed-forward": config([mamba(mlp=GLU)]),
    "attention": config([attention(mlp=None)]),
    "attention multi-head": config([attention(heads=3, kv_heads=3, dim=8, vdim=20, mlp=None)]),
    "attention one kv head": config([attention(heads=6, kv_heads=1, dim=40, vdim=12, chunk=7, mlp=None)]),
    "attention chunk of one": config([attention(chunk=1, mlp=None)]),
    "attention chunk longer than the sequence": config([attention(chunk=1000, mlp=None)]),
    "attention with feed-forward": config([attention()]),
    "feed-forward odd width": config([attention(mlp={"kind": "dense", "ff": 27, "limit": 2.5})]),
    "one stream": config([mamba(), attention()], streams=1),
    "two streams": config([mamba(), attention()], streams=2),
    "six streams": config([mamba(), attention()], streams=6),
    "one norm group": config([attention()], groups=1),
    "many norm groups": config([attention(), mamba()], groups=20, width=80),
    "no input convolution reach": config([attention(), mamba()], taps=1),
    "long input convolution": config([attention(), mamba()], taps=6),
    "odd width": config([attention(), mamba(heads=3, vdim=5, groups=1, norm_groups=3)], width=57, groups=3, vocab=61),
    "layers of different sizes": config([mamba(), attention(), mamba(heads=2, vdim=24, state=40, groups=1, conv=2, norm_groups=1),
                                         attention(heads=2, kv_heads=1, dim=16, vdim=32, chunk=5, mlp=None), mamba(mlp={"kind": "dense", "ff": 24, "limit": 1.5})]),
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
        _cache[key] = (w, t, *ho.forward(cfg, values(w), t))
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
    assert m.seq_len() == n
    m.destroy()


MIXED = config([mamba(), attention(chunk=16), mamba(heads=2, vdim=32, state=32, groups=1, norm_groups=2, mlp=GLU), attention(chunk=11)], taps=4)


@pytest.mark.parametrize("max_rows", [0, 5])
@pytest.mark.parametrize("cuts", [[2] * 40, [1, 2, 3, 5, 7, 11, 13, 17, 21], [16, 16, 16, 32], [15, 2, 30, 2, 31], [79, 1]])
def test_portions(dev, cuts, max_rows):
    """Whatever the portions (and the rows of a block inside them), every position has the same logits."""
    n = sum(cuts)
    w, t, logits, _ = oracle("mixed", MIXED, n)
    m = build(dev, MIXED, w, n, max_rows=max_rows)
    got, at = [], 0
    for c in cuts:
        got.append(m.extend(t[at:at + c], range(c)))
        at += c
    check(np.concatenate(got), logits, F32_TOL)
    m.destroy()


@pytest.mark.parametrize("dtype,tol", [("float32", F32_TOL), ("bfloat16", BF16_TOL)])
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


def test_wanted_places_only(dev):
    n = 30
    w, t, logits, _ = oracle("mixed", MIXED, n)
    m = build(dev, MIXED, w, n, max_rows=7)
    want = [0, 6, 7, 13, 29]
    check(m.extend(t, want), logits[want], F32_TOL)
    with pytest.raises(Exception):
        m.extend(t[:1])  # beyond max_seq
    m.destroy()


def test_batch_of_unequal_sequences(dev):
    """Sequences decoded side by side (prompts of different lengths, in different places of their chunks) equal each alone."""
    cfg, lens, steps = MIXED, [1, 2, 15, 40], 19
    w = weights(cfg)
    seqs = [tokens(cfg, n + steps, seed=i) for i, n in enumerate(lens)]
    refs = [ho.forward(cfg, values(w), s)[0] for s in seqs]
    for dtype, tol in (("float32", F32_TOL), ("bfloat16", BF16_TOL)):
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


def test_slots_are_reused(dev):
    """A freed slot's K/V rows, recurrent state and histories do not reach the next sequence, short or long."""
    cfg = MIXED
    w = weights(cfg)
    m = build(dev, cfg, w, 64, max_batch=2)
    for seed, n in enumerate([50, 1, 3, 29, 2]):
        t = tokens(cfg, n, seed)
        ref = ho.forward(cfg, values(w), t)[0]
        for slot in (1, 0):
            m.release(slot)
            check(m.extend(t, range(n), seq=slot), ref, F32_TOL)
        m.release(0)
        for i in range(n):  # and through the decode step
            m.decode([t[i]], 1)
            assert row_errors(m.read_logits(cfg["vocab"]), ref[i]) < F32_TOL
    m.destroy()


# ---- keys at a chunk's edge, far and near ---------------------------------------------------------
def _edge_model(chunk, dim=16, scale=6.0):
    """Attention reads the token itself (no reach of the input convolution) and one key stands out: every query points at
    token 1's key, whose value is large."""
    cfg = config([attention(heads=2, kv_heads=1, dim=dim, vdim=dim, scale=scale, chunk=chunk, mlp=None)], width=32, taps=1, streams=2, groups=1, vocab=40)
    w = values(weights(cfg, 3))
    from doppler_b200.safetensors import bf16_bits
    e = np.zeros((40, 32))
    e[:, 0] = 1.0                      # every token's query direction
    e[1:, 1] = np.where(np.arange(1, 40) == 1, 1.0, -1.0)
    e[:, 2:] = np.random.default_rng(5).standard_normal((40, 30)) * 0.3
    e[1, 2:] *= 4.0
    w["embed"] = e
    q, k = np.zeros((2 * dim, 32)), np.zeros((dim, 32))
    q[[0, dim], 0] = 1.0
    k[0, 1] = 1.0
    k[1:, 2:2 + dim - 1] = 0.02 * np.random.default_rng(6).standard_normal((dim - 1, dim - 1))
    q[1:dim, 2:2 + dim - 1] = 0.02
    w["l0.mix.q"], w["l0.mix.k"] = q, k
    return cfg, {n: bf16_bits(v) for n, v in w.items()}


@pytest.mark.parametrize("dim,dtype,tol", [(16, "float32", F32_TOL), (16, "bfloat16", BF16_TOL), (64, "bfloat16", BF16_TOL), (128, "bfloat16", BF16_TOL)])
@pytest.mark.parametrize("chunk", [32, 33, 96, 200])
def test_chunk_edges(dev, chunk, dim, dtype, tol):
    """The standing-out key at the first place of a chunk, and at the last place of the chunk before: just inside and just
    outside for every query of the chunk, in prompts, in portions cut at and around the edge, and in decoding."""
    if dim > 30:
        cfg = config([attention(heads=4, kv_heads=2, dim=dim, vdim=dim, scale=0.6, chunk=chunk, mlp=None)], width=32, taps=1, streams=2, groups=1, vocab=40)
        w = weights(cfg, 3)
    else:
        cfg, w = _edge_model(chunk, dim)
    v = values(w)
    n = 2 * chunk + 9
    for place in (chunk - 1, chunk, 2 * chunk - 1, 2 * chunk):
        t = 2 + tokens(cfg, n, 4) % 38
        t[place] = 1
        ref = ho.forward(cfg, v, t)[0]
        m = build(dev, cfg, w, n, dtype=dtype)
        check(m.extend(t, range(n)), ref, tol)
        m.release(0)
        cut = chunk + (place % 3) - 1
        a, b = m.extend(t[:cut], range(cut)), m.extend(t[cut:n - 12], range(n - 12 - cut))
        check(np.concatenate([a, b]), ref[:n - 12], tol)
        for i in range(n - 12, n):  # decoding over the second edge
            m.decode([t[i]], 1)
            assert row_errors(m.read_logits(), ref[i]) < tol
        m.destroy()


def test_tokens_of_other_chunks_do_not_reach(dev):
    """Exactly: with no convolution reach, what a chunk computes does not depend on the tokens before it."""
    chunk, n = 24, 60
    cfg, w = _edge_model(chunk)
    t = 2 + tokens(cfg, n, 9) % 38
    u = t.copy()
    u[chunk - 1] = 1
    m = build(dev, cfg, w, n)
    a = m.extend(t, range(n))
    m.release(0)
    b = m.extend(u, range(n))
    m.destroy()
    assert np.array_equal(a[chunk:], b[chunk:]) and not np.allclose(a[chunk - 1], b[chunk - 1], atol=1e-3)


def test_long_decoding(dev):
    """Several hundred decode steps: recurrent state, many chunks, and the split of a long chunk's keys."""
    cfg = config([mamba(state=32), attention(dim=16, vdim=24, chunk=300), mamba(vdim=20, heads=2, groups=1), attention(chunk=37)])
    n, pre = 420, 3
    w, t, logits, _ = oracle("long", cfg, n)
    m = build(dev, cfg, w, n)
    m.extend(t[:pre])
    errs = []
    for i in range(pre, n):
        m.decode([t[i]], 1)
        errs.append(row_errors(m.read_logits(), logits[i]))
    assert max(errs) < 2 * F32_TOL
    m.destroy()


# ---- the kernels of the larger sizes (bf16) --------------------------------------------------------
LARGE = {
    # tensor-core attention (head sizes 64 and 128, several group ratios), chunks shorter and longer than a split
    "attention 128": config([attention(heads=8, kv_heads=2, dim=128, vdim=128, scale=0.2, chunk=150)], width=128),
    "attention 128 mha": config([attention(heads=2, kv_heads=2, dim=128, vdim=128, scale=0.2, chunk=64)], width=128),
    "attention 64": config([attention(heads=8, kv_heads=1, dim=64, vdim=64, scale=0.3, chunk=1000)], width=128),
    "attention 64 and 128": config([attention(heads=4, kv_heads=2, dim=64, vdim=128, scale=0.3, chunk=90)], width=128),
    # recurrence in chunks: every column block and state size
    "ssm 128 x 64": config([mamba(heads=100, vdim=64, state=128, groups=4, norm_groups=4)], width=128),
    "ssm 64 x 32": config([mamba(heads=96, vdim=32, state=64, groups=3, norm_groups=3)], width=128),
    "ssm 32 x 16": config([mamba(heads=6, vdim=16, state=32, groups=2, norm_groups=2)], width=128),
    "ssm 128 x 16": config([mamba(heads=2, vdim=48, state=128, groups=1, norm_groups=2)], width=128),
    "ssm 64 x 16": config([mamba(heads=2, vdim=16, state=64, groups=2, norm_groups=1)], width=128),
    "ssm 32 x 32": config([mamba(heads=48, vdim=64, state=32, groups=2, norm_groups=2)], width=128),
    "ssm 32 x 64": config([mamba(heads=90, vdim=64, state=32, groups=2, norm_groups=2)], width=128),
    "ssm 64 x 64": config([mamba(heads=90, vdim=64, state=64, groups=2, norm_groups=2)], width=128),
    "ssm 128 x 32": config([mamba(heads=48, vdim=64, state=128, groups=2, norm_groups=2)], width=128),
    # products whose rows and columns do not fill a tile
    "wide": config([attention(heads=4, kv_heads=4, dim=72, vdim=56, mlp={"kind": "dense", "ff": 700, "limit": 1.0})], width=264, groups=3, vocab=600),
}


@pytest.mark.parametrize("name", LARGE)
def test_large_sizes_bf16(dev, name):
    """Prompts and portions around the 64-token chunks of the recurrence and the tiles of the products, then decoding."""
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


@pytest.mark.parametrize("heads,kv_heads,dim", [(8, 2, 128), (6, 2, 64), (12, 1, 64)])
def test_split_keys_bf16(dev, heads, kv_heads, dim):
    """A chunk so long that decoding splits its keys over several CTAs, before and after the chunk's edge."""
    cfg = config([attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, scale=0.25, chunk=640)], width=128)
    n = 660
    w, t, logits, _ = oracle(f"split {heads} {dim}", cfg, n)
    m = build(dev, cfg, w, 1300, dtype="bfloat16")
    got = [m.extend(t[:620], range(600, 620))]
    for i in range(620, n):
        m.decode([t[i]], 1)
        got.append(m.read_logits()[None])
    check(np.concatenate(got), logits[600:], BF16_TOL / 2)
    m.destroy()


def test_recurrence_in_chunks_is_32_bit(dev):
    """Inputs that bf16 holds exactly (one-hot projections of small integers, a convolution that passes its input through a
    saturated silu) leave only the recurrence's own arithmetic: chunks, token by token and the f32 mode agree closely."""
    cfg = config([mamba(heads=4, vdim=16, state=32, groups=1, conv=1, norm_groups=1)], width=128, taps=1, streams=1, groups=1, vocab=50, eps=1e-5)
    w = values(weights(cfg, 8))
    rng = np.random.default_rng(8)
    inner, ch = 64, 64 + 64
    w["embed"] = np.where(rng.random((50, 128)) < 0.5, 1.0, -1.0)   # unit root mean square: the norm divides by sqrt(9 + eps) after the scale
    w["l0.norm1"] = np.ones(128)
    w["l0.canon1"] = np.zeros((128, 1))
    p = np.zeros((inner + ch + 4, 128))
    p[np.arange(inner + ch), rng.integers(0, 128, inner + ch)] = 1.0
    w["l0.mix.in"] = p
    w["l0.mix.conv"] = np.full((ch, 1), 32.0)
    w["l0.mix.conv.b"] = np.full(ch, 64.0)                          # silu(64 +- 32) = 96 or 32
    w["l0.mix.A_log"] = np.array([-3.0, -1.0, 0.5, 1.5])
    w["l0.mix.dt_bias"] = np.array([-6.0, -5.0, -4.0, -2.0])
    from doppler_b200.safetensors import bf16_bits
    bits = {k: bf16_bits(v) for k, v in w.items()}
    n = 300
    t = tokens(cfg, n, 2)
    _, res = ho.forward(cfg, values(bits), t)
    y = {}
    for dtype in ("float32", "bfloat16"):
        m = build(dev, cfg, bits, n, dtype=dtype)
        m.extend(t)
        y[dtype] = m.read_hidden(n)
        m.destroy()
    check(y["float32"], res[-1], F32_TOL)
    # what is left in bf16: the output projection's operand
    assert row_errors(y["bfloat16"], res[-1]).max() < 4e-3


# ---- generation -------------------------------------------------------------------------------------
def _greedy(cfg, v, prompt, n):
    out = list(prompt)
    margins = []
    for _ in range(n):
        row = ho.forward(cfg, v, out)[0][-1]
        top = np.sort(row)[-2:]
        margins.append(top[1] - top[0])
        out.append(int(row.argmax()))
    return out[len(prompt):], min(margins)


@pytest.mark.parametrize("batch", [1, 3])
def test_greedy_generation(dev, tmp_path, batch):
    """Through the registry, the weight loading and the scheduler, from a model folder; prompts of different lengths, more of
    them than slots."""
    import json

    from doppler_b200.registry import load_model
    from doppler_b200.safetensors import write_bf16
    from doppler_b200.scheduler import Scheduler

    cfg = MIXED
    w = weights(cfg, 21)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    write_bf16(str(tmp_path / "model.safetensors"), w)
    prompts = [tokens(cfg, n, 30 + n).tolist() for n in (5, 1, 18, 33)]
    m = load_model(dev, str(tmp_path), 64, batch, "float32")
    got = Scheduler(m).generate(prompts, 24, block=7)
    stop = got[0][10]
    stopped = Scheduler(m).generate(prompts[:1], 24, stop=[stop])
    m.destroy()
    for p, toks in zip(prompts, got):
        want, margin = _greedy(cfg, values(w), p, 24)
        assert toks == want, (toks, want, margin)
    first = got[0].index(stop)
    assert stopped[0] == got[0][:first + 1]
    assert len(set(sum(got, []))) > 10, "decoding collapsed; the comparison would be vacuous"


def test_command_line_and_trace(dev, tmp_path):
    """`python -m doppler_b200 generate` and bin/trace_run, as a user starts them."""
    import json
    import os
    import subprocess
    import sys

    from doppler_b200.safetensors import write_bf16

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = MIXED
    w = weights(cfg, 21)
    model = tmp_path / "model"
    model.mkdir()
    (model / "config.json").write_text(json.dumps(cfg))
    write_bf16(str(model / "model.safetensors"), w)
    prompt = tokens(cfg, 9, 3).tolist()
    res = subprocess.run([sys.executable, "-m", "doppler_b200", "generate", "--model", str(model), "--prompt", ",".join(map(str, prompt)), "--max-new", "12",
                          "--dtype", "float32"], cwd=root, capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr
    assert json.loads(res.stdout.splitlines()[-1])["tokens"] == _greedy(cfg, values(w), prompt, 12)[0]

    t = tokens(cfg, 40, 4).tolist()
    ref = ho.forward(cfg, values(w), t)[0]
    short = tokens(cfg, 3, 5).tolist()
    ref2 = ho.forward(cfg, values(w), short)[0]
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": t[:30], "want": [0, 29, 7]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": t[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "a", "tokens": t[31:32], "want": [0]}], "end": []},
             {"step": 3, "entries": [{"id": "a", "tokens": t[32:], "want": [7]}], "end": ["a"]},
             {"step": 4, "entries": [{"id": "b", "tokens": short, "want": [0, 1, 2]}], "end": ["b"]}]
    out = tmp_path / "out"
    out.mkdir()
    res = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(model), "--dtype", "float32", "--out", str(out), "--max-tokens", "40"],
                         input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
    assert res.returncode == 0, res.stderr
    assert [l for l in res.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(5)]
    load = lambda i: np.fromfile(out / f"{i}.f32", "<f4").reshape(-1, cfg["vocab"])  # noqa: E731
    check(load(0), ref[[0, 29, 7]], F32_TOL)
    assert not (out / "1.f32").exists()
    check(load(2), ref[[31]], F32_TOL)
    check(load(3), ref[[39]], F32_TOL)
    check(load(4), ref2, F32_TOL)


def test_missing_and_misshapen_weights_are_refused(dev):
    from doppler_b200 import _lib as L
    from doppler_b200 import fenorax
    from doppler_b200.model import StackModel

    cfg = CASES["attention"]
    w = weights(cfg)
    stack, layers = fenorax.stack_config(cfg)
    m = StackModel(dev, stack, layers, 16)
    with pytest.raises(Exception, match="has not been loaded"):
        m.prefill([1, 2, 3])
    with pytest.raises(Exception, match="expects shape"):
        m.load_tensor(0, L.T_Q, w["l0.mix.q"][:, :-1].copy())
    with pytest.raises(Exception, match="has no"):
        m.load_tensor(0, L.T_SSM_IN, w["l0.mix.q"])
    m.destroy()
    with pytest.raises(Exception, match="heads over"):
        StackModel(dev, stack, [dict(layers[0], kv_heads=3)], 16)
