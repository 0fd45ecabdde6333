"""Fenorax without a GPU: the oracle, that the test weights make mistakes visible, configuration and weight files, the registry,
the scheduler and the trace replay (with a stand-in model)."""
import copy
import json

import numpy as np
import pytest

import hybrid_oracle as ho
from doppler_b200 import _lib as L
from doppler_b200 import fenorax, registry, trace
from doppler_b200.safetensors import SafetensorsError, SafetensorsFile, bf16_bits, bf16_values, write_bf16
from doppler_b200.scheduler import Scheduler
from fenorax_util import attention, config, mamba, row_errors, tokens, values, weights

CFG = config([mamba(), attention(chunk=16), mamba(heads=2, vdim=32, state=32, groups=1, norm_groups=2, mlp={"kind": "dense", "ff": 40, "limit": 0.75}),
              attention(chunk=11)], taps=4)
BF16_TOL, BF16_RMS = 8e-2, 3.5e-2  # the loosest tolerances of the GPU tests (largest row error, root mean square of the rows)


# ---- oracle -----------------------------------------------------------------------------------------
def test_oracle_recurrence_equals_its_unrolled_sum():
    rng = np.random.default_rng(0)
    T, H, P, N, G = 9, 4, 3, 5, 2
    x, B, C = rng.standard_normal((T, H, P)), rng.standard_normal((T, G, N)), rng.standard_normal((T, G, N))
    dt, A, D = rng.uniform(0.01, 1, (T, H)), rng.standard_normal(H), rng.standard_normal(H)
    y = ho.ssd_scan(x, B, C, dt, A, D)
    for h in range(H):
        g = h // (H // G)
        for t in range(T):
            want = D[h] * x[t, h]
            for s in range(t + 1):
                want = want + np.exp(-np.exp(A[h]) * dt[s + 1:t + 1, h].sum()) * dt[s, h] * (B[s, g] @ C[t, g]) * x[s, h]
            assert np.allclose(y[t, h], want)


def test_oracle_is_causal_and_prefix_consistent():
    w, t = values(weights(CFG)), tokens(CFG, 40)
    whole = ho.forward(CFG, w, t)[0]
    for n in (1, 2, 17, 33):
        assert np.allclose(ho.forward(CFG, w, t[:n])[0], whole[:n])


def _mistakes():
    yield "window one token short", lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=15)
    yield "window one token long", lambda c, w: c["layers"][1]["mixer"]["mask"].update(size=17)
    yield "other score scale", lambda c, w: c["layers"][1]["mixer"].update(scale=0.2)
    yield "norm not in groups", lambda c, w: c["norm"].update(groups=1)
    yield "embedding scale left out", lambda c, w: c["embedding"].update(scale=1.0)
    yield "clamp of the feed-forward", lambda c, w: c["layers"][1]["mlp"].update(limit=100.0)
    yield "recurrence norm not in groups", lambda c, w: c["layers"][0]["mixer"].update(norm_groups=1)

    def zero(name):
        return lambda c, w: w.update({name: np.zeros_like(w[name])})

    for name in ("l0.canon1", "l1.canon2", "l0.mix.conv.b", "l0.mix.D", "l0.mix.dt_bias", "l0.mix.A_log", "l1.mix.g", "l0.mix.conv"):
        yield "without " + name, zero(name)

    def transpose(name):
        return lambda c, w: w.update({name: w[name].T.copy()})

    yield "stream mix transposed", transpose("l1.hc1.mix")

    def reverse_taps(name):
        return lambda c, w: w.update({name: w[name][:, ::-1].copy()})

    yield "taps reversed", reverse_taps("l0.canon1")
    yield "convolution taps reversed", reverse_taps("l0.mix.conv")

    def swap_groups(c, w):  # heads dealt to the other group's B and C
        m = c["layers"][0]["mixer"]
        lo = m["heads"] * m["vdim"] * 2
        a = w["l0.mix.in"].copy()
        n = m["state"]
        a[[*range(lo, lo + 2 * n)]] = w["l0.mix.in"][[*range(lo + n, lo + 2 * n), *range(lo, lo + n)]]
        w["l0.mix.in"] = a

    yield "B of the other group", swap_groups


@pytest.mark.parametrize("name,plant", list(_mistakes()), ids=[n for n, _ in _mistakes()])
def test_mistakes_show(name, plant):
    """Every planted mistake moves some position's logits by more than the tolerances of the GPU tests."""
    w, t = values(weights(CFG)), tokens(CFG, 50)
    good = ho.forward(CFG, w, t)[0]
    cfg, bad = copy.deepcopy(CFG), dict(w)
    plant(cfg, bad)
    err = row_errors(ho.forward(cfg, bad, t)[0], good)
    assert err.max() > 2 * BF16_TOL or np.sqrt((err ** 2).mean()) > 1.3 * BF16_RMS


@pytest.mark.parametrize("dim", [16, 64, 128])
def test_chunk_edge_inputs_show_a_shifted_edge(dim):
    import test_gpu_fenorax as g

    chunk = 33
    if dim > 30:
        cfg = config([attention(heads=4, kv_heads=2, dim=dim, vdim=dim, scale=0.6, chunk=chunk, mlp=None)], width=32, taps=1, streams=2, groups=1, vocab=40)
        w = values(weights(cfg, 3))
    else:
        cfg, w = g._edge_model(chunk, dim)
        w = values(w)
    n = 2 * chunk + 9
    for place, off in ((chunk, 1), (2 * chunk, 1), (chunk - 1, -1), (2 * chunk - 1, -1)):
        t = 2 + tokens(cfg, n, 4) % 38
        t[place] = 1
        bad = copy.deepcopy(cfg)
        bad["layers"][0]["mixer"]["mask"]["size"] = chunk + off
        assert row_errors(ho.forward(bad, w, t)[0], ho.forward(cfg, w, t)[0]).max() > 2 * BF16_TOL


# ---- configuration and weights ------------------------------------------------------------------------
def test_stack_config_takes_everything_from_the_configuration():
    stack, layers = fenorax.stack_config(CFG)
    assert stack == {"width": 64, "vocab": 97, "streams": 3, "norm_groups": 2, "input_taps": 4, "eps": 1e-4, "embed_scale": 0.8}
    assert layers[0] == {"mixer": L.MIXER_MAMBA2, "heads": 4, "vdim": 16, "state": 16, "groups": 2, "conv_taps": 4, "norm_groups": 2}
    assert layers[1]["chunk"] == 16 and layers[1]["scale"] == 0.4 and layers[1]["ff"] == 40 and layers[1]["ff_limit"] == 0.75
    assert (layers[1]["ff_slope"], layers[1]["ff_shift"]) == (1.702, 1.0)
    assert "ff" not in layers[0] and layers[2]["ff"] == 40
    assert {n for n, _, _ in fenorax.model_tensors(layers)} == set(weights(CFG))


@pytest.mark.parametrize("change,text", [
    (lambda c: c.update(architecture="Other"), "is not Fenorax"),
    (lambda c: c.pop("streams"), "missing streams"),
    (lambda c: c["norm"].pop("eps"), "missing eps"),
    (lambda c: c["layers"][0].update(type="rwkv"), "unknown type"),
    (lambda c: c["layers"][1]["mixer"].pop("mask"), "missing mask"),
    (lambda c: c["layers"][1]["mlp"].update(kind="moe"), "unknown feed-forward"),
    (lambda c: c["layers"][1]["mlp"].update(limit=0), "must be positive"),
])
def test_bad_configurations_are_named(change, text):
    c = copy.deepcopy(CFG)
    change(c)
    with pytest.raises(fenorax.ConfigError, match=text):
        fenorax.stack_config(c)


def test_safetensors_round_trip(tmp_path):
    w = weights(CFG)
    path = str(tmp_path / "m.safetensors")
    write_bf16(path, w)
    f = SafetensorsFile(path)
    assert set(f.names()) == set(w) and "nothing" not in f
    for k, v in w.items():
        assert f.dtype(k) == "BF16" and np.array_equal(f.tensor(k), v)
    with pytest.raises(SafetensorsError, match="no tensor"):
        f.tensor("nothing")
    f.close()
    raw = bytearray(open(path, "rb").read())
    (tmp_path / "cut.safetensors").write_bytes(raw[:-2])
    cut = SafetensorsFile(str(tmp_path / "cut.safetensors"))
    with pytest.raises(SafetensorsError, match="do not hold"):
        cut.tensor(list(w)[-1])
    (tmp_path / "short.safetensors").write_bytes(b"\x01\x02")
    with pytest.raises(SafetensorsError, match="too short"):
        SafetensorsFile(str(tmp_path / "short.safetensors"))


def test_bf16_rounding():
    x = np.array([1.0, 1.00390625, 1.01171875, -3.14159, 1e-30, 0.0], np.float32)
    v = bf16_values(bf16_bits(x))
    assert v[0] == 1.0 and v[1] == 1.0 and v[2] == np.float32(1.015625)  # ties to even
    assert np.all(np.abs(v - x) <= np.abs(x) * 2.0 ** -8)


def test_registry(tmp_path):
    with pytest.raises(registry.UnknownModel, match="neither"):
        registry.describe(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps({"architecture": "Nobody"}))
    with pytest.raises(registry.UnknownModel, match="Nobody"):
        registry.describe(str(tmp_path))
    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert registry.describe(str(tmp_path)) == {"kind": "Fenorax", "config": CFG}
    with pytest.raises(ValueError, match="dtype"):
        registry.load_model(None, str(tmp_path), 8, dtype="int8")
    (tmp_path / "manifest.json").write_text("{}")
    assert registry.describe(str(tmp_path)) == {"kind": "rdrr"}


# ---- scheduler and trace --------------------------------------------------------------------------------
class FakeModel:
    """Runs 'next token = (sum of the sequence) % vocab' and keeps what the runner would keep."""

    def __init__(self, max_batch=1, vocab=11, max_seq=64):
        self.max_batch, self.cfg = max_batch, {"vocab": vocab, "max_seq": max_seq}
        self.seqs = [[] for _ in range(max_batch)]
        self.calls, self.last = [], None

    def _row(self, seq):
        return np.eye(self.cfg["vocab"], dtype=np.float32)[sum(seq) % self.cfg["vocab"]]

    def release(self, seq=0):
        self.seqs[seq] = []

    def seq_len(self, seq=0):
        return len(self.seqs[seq])

    def extend(self, tokens, want=(), seq=0):
        self.calls.append(("extend", seq, len(tokens)))
        assert list(want) == sorted(set(want))
        base = len(self.seqs[seq])
        self.seqs[seq] += list(tokens)
        return np.stack([self._row(self.seqs[seq][:base + w + 1]) for w in want]) if len(want) else np.empty((0, self.cfg["vocab"]), np.float32)

    def prefill(self, tokens, seq=0):
        return int(self.extend(tokens, [len(tokens) - 1], seq)[0].argmax())

    def decode(self, first, steps):
        self.calls.append(("decode", len(first), steps))
        out, cur = [], list(first)
        for _ in range(steps):
            for i, t in enumerate(cur):
                self.seqs[i].append(int(t))
            self.last = np.stack([self._row(self.seqs[i]) for i in range(len(cur))])
            cur = [int(r.argmax()) for r in self.last]
            out.append(cur)
        return np.array(out, np.int32)

    def read_logits(self, n):
        return self.last.ravel()[:n]


def test_scheduler_steps_and_slots():
    m = FakeModel(max_batch=2)
    s = Scheduler(m)
    a = s.step("a", [1, 2, 3], [2, 0])
    assert a.argmax(1).tolist() == [6, 1] and m.calls[-1] == ("extend", 0, 3)
    assert s.step("a", [4], [0]).argmax(1).tolist() == [10] and m.calls[-1] == ("decode", 1, 1)
    assert s.step("a", [1]).shape == (0, 11)
    assert s.step("b", [5], [0]).argmax(1).tolist() == [5] and m.calls[-1] == ("extend", 1, 1)  # a second sequence is alive
    with pytest.raises(RuntimeError, match="slots are taken"):
        s.step("c", [1])
    s.finish("a")
    s.finish("nobody")
    assert s.step("c", [7, 1], [1]).argmax(1).tolist() == [8] and m.calls[-1] == ("extend", 0, 2)  # a's slot, from position 0
    with pytest.raises(ValueError):
        s.step("c", [7], [1])


def _fake_greedy(prompt, n, vocab=11):
    seq = list(prompt)
    for _ in range(n):
        seq.append(sum(seq) % vocab)
    return seq[len(prompt):]


@pytest.mark.parametrize("batch", [1, 2, 4])
def test_scheduler_generates(batch):
    prompts = [[1, 2], [3], [5, 5, 5]]
    for n in (0, 1, 9):
        got = Scheduler(FakeModel(max_batch=batch)).generate(prompts, n, block=4)
        assert got == [_fake_greedy(p, n) for p in prompts]
    full = _fake_greedy([1, 2], 30)
    cut = Scheduler(FakeModel()).generate([[1, 2]], 30, stop=[full[5]], block=4)[0]
    assert cut == full[:full.index(full[5]) + 1]
    assert len(Scheduler(FakeModel(max_seq=10)).generate([[1, 2]], 30)[0]) == 9  # the cache ends it


def test_trace_steps(tmp_path):
    s = Scheduler(FakeModel())
    trace.run_step(s, {"step": 0, "entries": [{"id": "x", "tokens": [1, 2, 3], "want": [0, 2]}], "end": []}, str(tmp_path))
    trace.run_step(s, {"step": 1, "entries": [{"id": "x", "tokens": [4], "want": []}], "end": ["x"]}, str(tmp_path))
    trace.run_step(s, {"step": 2, "entries": [{"id": "y", "tokens": [9], "want": [0]}], "end": ["y"]}, str(tmp_path))
    assert np.fromfile(tmp_path / "0.f32", "<f4").reshape(2, 11).argmax(1).tolist() == [1, 6]
    assert np.fromfile(tmp_path / "2.f32", "<f4").argmax() == 9
    assert sorted(p.name for p in tmp_path.iterdir()) == ["0.f32", "2.f32"]


def test_command_line_info(tmp_path, capsys):
    from doppler_b200 import __main__ as cli

    (tmp_path / "config.json").write_text(json.dumps(CFG))
    assert cli.info(["--model", str(tmp_path)]) == 0
    d = json.loads(capsys.readouterr().out)
    assert d["kind"] == "Fenorax" and len(d["layers"]) == 4
