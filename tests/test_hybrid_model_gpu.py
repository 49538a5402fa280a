"""Hybrid decoders (models::HybridLM behind the registry) on the GPU against the plain model of hybrid_reference.py; limits as in
sequence_check.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import sequence_check
from hybrid_cases import CASES, ReferenceHybrid, build, reference, save, weights
from sequence_check import errors, run, status

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_cache = {}


def Sequence(c, w, ids, **kw):
    return sequence_check.Sequence(ReferenceHybrid, c, w, ids, **kw)


def case(name):
    """(config, weights, one sequence) of a configuration."""
    if name not in _cache:
        c = CASES[name]
        w = weights(c, seed=len(name))
        _cache[name] = (c, w, Sequence(c, w, np.random.default_rng(1).integers(0, c["vocab"], 170)))
    return _cache[name]


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CASES))
def test_prompts_portions_and_tokens(cuda, name, dtype):
    c, w, q = case(name)
    m = build(c, w, dtype, max_seq_len=200)
    L = len(q.ids)
    q.check(run(m, q.ids, [L]), dtype)
    portions = [2, 3, 64, 1, 2, 30, 1, 1, 5]
    q.check(run(m, q.ids, portions + [L - sum(portions)]), dtype)
    q.check(run(m, q.ids, [L - 60] + [1] * 60), dtype)
    q.check(run(m, q.ids[:40], [1] * 40), dtype)
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_residual_stream_after_every_layer_execution(cuda, dtype):
    c, w, q = case("looped")
    m = build(c, w, dtype, max_seq_len=200)
    m.init_cache(1)
    taps = []
    reference(c, w).forward(q.ids[:50], taps)
    y, got = m.forward_tapped(q.ids[None, :50], 0, c["width"])       # the loop's additions as launches of their own
    q.check(y[0], dtype)
    assert got.shape[0] == len(taps) == 1 + 2 * 3 + 1
    for i, t in enumerate(taps):
        assert errors(got[i, 0], t).max() <= (1e-5 if dtype == "float32" else 4e-2), i
    m.init_cache(1)
    q.check(m.forward_with_cache(q.ids[None, :50], 0)[0], dtype)     # and inside the projections before them
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["looped", "ragged"])
def test_sequences_interleave_and_slots_are_reused(cuda, name, dtype):
    c, w, _ = case(name)
    rng = np.random.default_rng(5)
    qa, qb, qd = (Sequence(c, w, rng.integers(0, c["vocab"], n)) for n in (70, 33, 90))
    m = build(c, w, dtype, max_seq_len=200, max_sequences=3)
    a, b = m.open_sequence(), m.open_sequence()
    qa.check(m.extend(a, qa.ids[:40]), dtype)
    qb.check(m.extend(b, qb.ids), dtype)
    qa.check(m.extend(a, qa.ids[40:41]), dtype, 40)
    m.close_sequence(b)                               # b's slot goes to a longer sequence
    d = m.open_sequence()
    assert d == b
    for at in range(3):
        qd.check(m.extend(d, qd.ids[at:at + 1]), dtype, at)
        qa.check(m.extend(a, qa.ids[41 + at:42 + at]), dtype, 41 + at)
    qd.check(m.extend(d, qd.ids[3:]), dtype, 3)
    qa.check(m.extend(a, qa.ids[44:]), dtype, 44)
    m.open_sequence()
    with pytest.raises(RuntimeError, match="in use"):
        m.open_sequence()
    status()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_batches_against_each_alone(cuda, dtype):
    c, w, _ = case("tail")
    ids = np.random.default_rng(6).integers(0, c["vocab"], (5, 66))
    qs = [Sequence(c, w, r) for r in ids]
    m = build(c, w, dtype, max_seq_len=200)
    m.init_cache(5)
    at = 0
    for n in (40, 2, 1, 1, 20, 1, 1):
        y = m.forward_with_cache(ids[:, at:at + n], at)
        for b in range(5):
            qs[b].check(y[b], dtype, at)
        at += n
    with pytest.raises(RuntimeError, match="does not stand at"):
        m.forward_with_cache(ids[:, :1], 3)
    y = m.forward_with_cache(ids[:3, :30], 0, last_only=True)         # position 0 starts new sequences in used slots
    for b in range(3):
        qs[b].check(y[b], dtype, 29)
    status()
    m.close()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding(cuda, dtype):
    """Hundreds of single tokens: ring wraps, taps wrap, the state carries on."""
    c, w, _ = case("looped")
    if "long" not in _cache:
        _cache["long"] = Sequence(c, w, np.random.default_rng(7).integers(0, c["vocab"], 420), trials=2)
    q = _cache["long"]
    m = build(c, w, dtype, max_seq_len=500)
    q.check(run(m, q.ids, [5] + [1] * 415), dtype)
    m.close()


@pytest.mark.parametrize("use_graph", [True, False])
@pytest.mark.parametrize("name,dtype", [("looped", "bfloat16"), ("ragged", "bfloat16"), ("tail", "float32"), ("recurrent", "float32"), ("once", "bfloat16")])
def test_greedy_generation(cuda, name, dtype, use_graph):
    """Generator on a batch of prompts: every token an arg-max of the reference's logits for the same history."""
    c, w, q = case(name)
    B, P, n = 3, 37, 40
    prompt = np.random.default_rng(8).integers(0, c["vocab"], (B, P)).astype(np.int32)
    m = build(c, w, dtype, max_seq_len=200)
    toks, t = m.generate_greedy(prompt, n, use_graph=use_graph)
    assert toks.shape == (B, P + n) and np.array_equal(toks[:, :P], prompt) and t["graph_replay"] == use_graph
    for b in range(B):
        want = reference(c, w).forward(toks[b, :-1])[P - 1:]
        slack = 2 * np.sqrt(2 * np.log(c["vocab"])) * q.limits[dtype].max() * q.rms
        picked = want[np.arange(n), toks[b, P:]]
        assert (picked >= want.max(-1) - slack).all()
    again, _ = m.generate_greedy(prompt, n, use_graph=use_graph)      # the same cache memory, another run
    assert np.array_equal(again, toks)
    stop = int(toks[0, P + 3])
    short, _ = m.generate_greedy(prompt[:1], n, stop_ids=[stop], use_graph=use_graph)
    first = P + int(np.argmax(toks[0, P:] == stop))
    assert short.shape[1] == first + 1 and np.array_equal(short[0], toks[0, :first + 1])
    status()
    m.close()


def test_model_folder_registry_and_errors(cuda, tmp_path):
    from vesper_b200.model import load_model
    c, w, q = case("tail")
    ids = q.ids
    save(tmp_path, c, w)
    m = load_model(str(tmp_path), "float32", max_seq_len=200)
    q.check(run(m, ids[:50], [50]), "float32")
    with pytest.raises(RuntimeError, match="exceeds maximum"):
        run(m, np.concatenate([ids, ids]), [2 * len(ids)])
    m.close()
    save(tmp_path, c, {k: v for k, v in w.items() if k != "l1.mix.sink"})
    with pytest.raises(RuntimeError, match="l1.mix.sink"):
        load_model(str(tmp_path))
    save(tmp_path, c, dict(w, bigram=w["bigram"][:-1]))
    with pytest.raises(RuntimeError, match="bigram"):
        load_model(str(tmp_path))


def test_transformer_checkpoint_through_the_registry(cuda, tmp_path):
    """The Llama-style decoder loads from a folder too, and equals the model whose parameters are set one by one."""
    from helpers import model_weights
    from vesper_b200.model import TransformerLM, load_model, param_shapes
    cfg = dict(vocab=160, dim=256, n_layers=2, n_heads=2, n_kv_heads=1, ffn_hidden=320)
    w = model_weights(param_shapes(**cfg), 3, std=0.06)
    from helpers import bf16_round
    w = {k: bf16_round(v) for k, v in w.items()}
    save(tmp_path, dict(architecture="TransformerLM", vocab_size=160, dim=256, n_layers=2, n_heads=2, n_kv_heads=1, ffn_hidden_dim=320, max_seq_len=64, norm_eps=1e-6), w)
    m = load_model(str(tmp_path))
    t = TransformerLM(160, 256, 2, 2, 1, 320, 64)
    for k, v in w.items():
        t.set_param(k, v)
    ids = np.random.default_rng(2).integers(0, 160, 20)
    got = run(m, ids, [12, 1, 1, 6])
    t.init_cache(1)
    assert errors(got, t.forward_with_cache(ids[None], 0)[0]).max() <= 2e-2
    m.close(); t.close()


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(cuda, tmp_path, dtype):
    c, w, q = case("looped")
    save(tmp_path, c, w)
    ids, other = q.ids, np.random.default_rng(9).integers(0, c["vocab"], 25)
    q2 = Sequence(c, w, other)
    steps = [dict(entries=[dict(id="a", tokens=ids[:60].tolist(), want=[0, 59, 7])], end=[]),
             dict(entries=[dict(id="b", tokens=other[:2].tolist(), want=[])], end=[]),
             dict(entries=[dict(id="a", tokens=ids[60:61].tolist(), want=[0]), dict(id="b", tokens=other[2:].tolist(), want=[22, 1])], end=["a"]),
             dict(entries=[dict(id="c", tokens=ids[:3].tolist(), want=[2])], end=["b", "c"])]
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "200"],
                       input=text, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert r.stdout.split("\n")[:4] == ["done 0", "done 1", "done 2", "done 3"]
    rows = {0: [(q, 0), (q, 59), (q, 7)], 2: [(q, 60), (q2, 24), (q2, 3)], 3: [(q, 2)]}
    assert not (tmp_path / "1.f32").exists()
    for i, x in rows.items():
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(len(x), c["vocab"])
        for y, (seq, at) in zip(got, x):
            seq.check(y[None], dtype, at)


def test_generate_command(cuda, tmp_path):
    c, w, _ = case("tail")
    save(tmp_path, c, w)
    r = subprocess.run([sys.executable, "-m", "vesper_b200.generate", "--model", str(tmp_path), "--new", "6", "--prompt", "5 9 2", "--prompt", "1 1 7"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [[int(t) for t in line.split()] for line in r.stdout.strip().splitlines()]
    m = build(c, w, "bfloat16", max_seq_len=200)
    assert np.array_equal(m.generate_greedy(np.array([[5, 9, 2], [1, 1, 7]]), 6)[0], np.array(lines))
    m.close()
