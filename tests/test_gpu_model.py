"""Whole-model parity: the CUDA runner against the oracle model on the same seeded weights.
Gate: greedy decode token-identical for 64 tokens."""
import json
import os

import numpy as np
import pytest

from doppler_b200 import synthetic
from doppler_b200.model import DecoderModel
from model_util import gaussian_model_weights
from oracle import oracle as O
from parity import assert_close

pytestmark = pytest.mark.gpu
GOLDEN = os.path.join(os.path.dirname(os.path.abspath(__file__)), "golden")


def _weights(cfg, kind, seed):
    """'blocks': the benchmark generator (uniform random Q4_K blocks, as BASELINE config 0 specifies);
    'gaussian': quantised zero-mean gaussians (decoding visits many tokens)."""
    return synthetic.make_model_weights(cfg, seed=seed) if kind == "blocks" else gaussian_model_weights(cfg, seed)


def _run_pair(dev, name, prompt_len, steps, max_seq, kind="gaussian"):
    cfg = dict(synthetic.MODEL_CONFIGS[name])
    w = _weights(cfg, kind, 1234)
    prompt = synthetic.make_prompt(cfg, prompt_len, seed=1234)
    m = DecoderModel(dev, cfg, max_seq=max_seq)
    m.load_all(w)
    first = m.prefill(prompt)
    logits_gpu = m.read_logits()
    cfg_o = dict(cfg, max_seq=max_seq)
    om = O.OracleModel(cfg_o, w)
    tok, margin, logits_cpu = om.forward(prompt, want_logits=True)
    assert_close(logits_gpu, logits_cpu, f"{name}: prefill logits")
    assert first == tok, f"{name}: prefill token {first} vs oracle {tok} (oracle margin {margin:.3e})"
    out = m.decode([first], steps)[:, 0]
    cur = tok
    for s in range(steps):
        nxt, margin = om.forward([cur])
        assert int(out[s]) == nxt, f"{name}: step {s}: GPU token {int(out[s])} vs oracle {nxt} (oracle margin {margin:.3e})"
        cur = nxt
    assert m.seq_len() == prompt_len + steps
    m.destroy()
    if kind == "gaussian":
        assert len(set(out.tolist())) > steps // 4, "decoding collapsed; the identity check would be vacuous"
    return out


@pytest.mark.parametrize("kind", ["gaussian", "blocks"])
def test_tiny_model_tokens_identical(dev, kind):
    _run_pair(dev, "tiny", prompt_len=24, steps=64, max_seq=128, kind=kind)


def test_small_model_tokens_identical(dev):
    """Three layers at the 0.6B shape (hidden 1024, 16/8 heads, D 128, MLP 3072), vocabulary 4096."""
    _run_pair(dev, "small", prompt_len=40, steps=64, max_seq=128, kind="gaussian")


def test_small_model_long_context_split_attention(dev):
    """max_seq 1024 makes the decode attention split the KV range, which takes the fused
    split-merge + activation-digit kernel on the way to o_proj."""
    _run_pair(dev, "small", prompt_len=300, steps=64, max_seq=1024, kind="gaussian")


def test_small_model_benchmark_blocks(dev):
    _run_pair(dev, "small", prompt_len=40, steps=64, max_seq=128, kind="blocks")


def test_golden_tokens(dev):
    """Committed fixture made by tests/golden/make_golden.py from the oracle."""
    g = json.load(open(os.path.join(GOLDEN, "model_tokens.json")))
    cfg = dict(synthetic.MODEL_CONFIGS[g["config"]])
    m = DecoderModel(dev, cfg, max_seq=g["max_seq"])
    m.load_all(gaussian_model_weights(cfg, g["seed"]))
    prompt = synthetic.make_prompt(cfg, g["prompt_len"], seed=g["seed"])
    assert prompt.tolist() == g["prompt"]
    first = m.prefill(prompt)
    assert first == g["tokens"][0]
    out = m.decode([first], len(g["tokens"]) - 1)[:, 0]
    assert out.tolist() == g["tokens"][1:]
    m.destroy()


def test_decode_resumes_and_resets(dev):
    cfg = dict(synthetic.MODEL_CONFIGS["tiny"])
    w = gaussian_model_weights(cfg, 99)
    prompt = synthetic.make_prompt(cfg, 16, seed=99)
    m = DecoderModel(dev, cfg, max_seq=96)
    m.load_all(w)
    first = m.prefill(prompt)
    a = m.decode([first], 40)[:, 0]
    m.reset()
    first2 = m.prefill(prompt)
    b1 = m.decode([first2], 15)[:, 0]
    b2 = m.decode([int(b1[-1])], 25)[:, 0]  # continuing in a second call gives the same stream
    assert first == first2 and np.array_equal(a, np.concatenate([b1, b2]))
    with pytest.raises(Exception):
        m.decode([0], 1000)  # beyond max_seq
    m.destroy()


def test_batched_decode_is_independent_sequences(dev):
    """Batch is an extension of the reference (which decodes one sequence): its oracle is the
    same number of independent single-sequence runs.  Different prompt lengths per sequence."""
    cfg = dict(synthetic.MODEL_CONFIGS["small"])
    w = gaussian_model_weights(cfg, 4321)
    lens = [33, 7, 64, 20]
    steps, max_seq = 24, 128
    m = DecoderModel(dev, cfg, max_seq=max_seq, max_batch=len(lens))
    m.load_all(w)
    prompts = [synthetic.make_prompt(cfg, n, seed=4321, seq=i) for i, n in enumerate(lens)]
    firsts = [m.prefill(p, seq=i) for i, p in enumerate(prompts)]
    out = m.decode(firsts, steps)  # [steps, batch]
    assert out.shape == (steps, len(lens))
    for i, p in enumerate(prompts):
        om = O.OracleModel(dict(cfg, max_seq=max_seq), w)
        tok, margin = om.forward(p)
        assert firsts[i] == tok, f"sequence {i}: prefill token {firsts[i]} vs oracle {tok} (margin {margin:.3e})"
        cur = tok
        for s in range(steps):
            cur, margin = om.forward([cur])
            assert int(out[s, i]) == cur, f"sequence {i} step {s}: {int(out[s, i])} vs oracle {cur} (margin {margin:.3e})"
        assert m.seq_len(i) == lens[i] + steps
    m.destroy()


def test_portions_return_the_same_logits(dev):
    """dp_model_extend: a prompt in portions, logits at wanted places, against whole prompts."""
    cfg = dict(synthetic.MODEL_CONFIGS["tiny"])
    m = DecoderModel(dev, cfg, max_seq=96)
    m.load_all(gaussian_model_weights(cfg, 7))
    prompt = synthetic.make_prompt(cfg, 40, seed=7)
    assert m.extend(prompt[:9]).shape == (0, cfg["vocab"])
    rows = m.extend(prompt[9:], [0, 12, 30])
    for place, row in zip((9, 21, 39), rows):
        m.reset()
        m.prefill(prompt[:place + 1])
        assert_close(row, m.read_logits(), f"logits at {place}")
    m.destroy()


def test_artifact_through_the_registry_and_scheduler(dev, tmp_path):
    """An RDRR folder opened by the model registry and run by the scheduler gives the runner's own greedy tokens."""
    from doppler_b200.rdrr import write_artifact
    from doppler_b200.registry import load_model
    from doppler_b200.scheduler import Scheduler

    cfg = dict(synthetic.MODEL_CONFIGS["tiny"])
    w = gaussian_model_weights(cfg, 11)
    w["layers"] = [{k: v.astype(np.float16).astype(np.float32) if k.endswith("norm") else v for k, v in l.items()} for l in w["layers"]]
    w["final_norm"] = w["final_norm"].astype(np.float16).astype(np.float32)
    write_artifact(str(tmp_path), dict(cfg, max_seq_len=256), w)
    prompts = [synthetic.make_prompt(cfg, n, seed=11, seq=n).tolist() for n in (12, 5)]
    m = load_model(dev, str(tmp_path), 96, max_batch=2)
    got = Scheduler(m).generate(prompts, 20, block=6)
    m.destroy()
    m = DecoderModel(dev, cfg, max_seq=96, max_batch=2)
    m.load_all(w)
    firsts = [m.prefill(p, seq=i) for i, p in enumerate(prompts)]
    out = m.decode(firsts, 19)
    m.destroy()
    assert got == [[f, *out[:, i].tolist()] for i, f in enumerate(firsts)]
