"""Zudisun decoders (models::HybridLM behind the registry) on the GPU against the plain model of zudisun_reference.py; limits as in
sequence_check.py."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest

import sequence_check
from sequence_check import errors, run, status
from zudisun_cases import CASES, attention, build, config, dense, mamba, moe, reference, save, weights

pytestmark = pytest.mark.gpu

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
_cache = {}
DTYPES = ["float32", "bfloat16"]


def Sequence(c, w, ids, **kw):
    return sequence_check.Sequence(reference, c, w, ids, **kw)


def case(name):
    """(config, rows of the bias tables, weights, one sequence) of a configuration."""
    if name not in _cache:
        c, rel = CASES[name]
        w = weights(c, rel, seed=len(name))
        _cache[name] = (c, rel, w, Sequence(c, w, np.random.default_rng(1).integers(0, c["vocab"], 150), trials=4))
    return _cache[name]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(CASES))
def test_prompts_portions_and_tokens(cuda, name, dtype):
    c, rel, w, q = case(name)
    m = build(c, rel, w, dtype, max_seq_len=160)
    L = len(q.ids)
    q.check(run(m, q.ids, [L]), dtype)
    portions = [2, 3, 64, 1, 2, 30, 1, 1, 5]
    q.check(run(m, q.ids, portions + [L - sum(portions)]), dtype)
    q.check(run(m, q.ids, [2] * (L // 2)), dtype)
    q.check(run(m, q.ids, [L - 60] + [1] * 60), dtype)
    q.check(run(m, q.ids[:40], [1] * 40), dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "ragged"])
def test_residual_stream_after_every_layer(cuda, name, dtype):
    c, rel, w, q = case(name)
    m = build(c, rel, w, dtype, max_seq_len=160)
    m.init_cache(1)
    taps = []
    reference(c, w).forward(q.ids[:50], taps)
    y, got = m.forward_tapped(q.ids[None, :50], 0, c["width"])
    q.check(y[0], dtype)
    assert got.shape[0] == len(taps) == len(c["layers"])
    for i, t in enumerate(taps):
        e = errors(got[i, 0], t)
        assert (e.max() <= 1e-5) if dtype == "float32" else (np.median(e) <= 2e-2), (i, e.max())
    m.close()


def test_every_mechanism_shows_in_the_logits(cuda):
    """A weight of each mechanism changed on one side only is far outside the limits (so the comparisons above see it)."""
    c, rel, w, q = case("mixed")
    m = build(c, rel, w, "float32", max_seq_len=160)
    for name, change in (("l0.mix.rel", lambda v: np.roll(v, 1, axis=0)), ("l0.mix.talk", np.transpose), ("l2.mix.pb", lambda v: v + 0.05), ("l2.mix.vmix", lambda v: v * 0.8),
                         ("l4.mix.g", lambda v: v * 0.9), ("l1.mix.D", lambda v: v + 0.05), ("l1.mix.dt.b", lambda v: v + 0.05), ("l3.mix.A_log", lambda v: v + 0.05),
                         ("l1.mlp.correction", lambda v: v[::-1]), ("l0.mlp.gate.b", lambda v: v + 0.05), ("l4.norm2", lambda v: v * 1.01), ("l3.mix.conv", lambda v: v[:, ::-1])):
        other = reference(c, dict(w, **{name: np.array(change(w[name]))})).forward(q.ids[:100])
        e = errors(q.want[:100], other)
        assert e.max() > 20 * 1e-4, (name, e.max())
    q.check(run(m, q.ids, [100, 50]), "float32")
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["mixed", "ragged"])
def test_sequences_interleave_and_slots_are_reused(cuda, name, dtype):
    c, rel, w, _ = case(name)
    rng = np.random.default_rng(5)
    qa, qb, qd = (Sequence(c, w, rng.integers(0, c["vocab"], n), trials=3) for n in (70, 33, 90))
    m = build(c, rel, w, dtype, max_seq_len=100, max_sequences=3)
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
    with pytest.raises(RuntimeError, match="exceeds maximum"):
        m.extend(d, np.zeros(11, np.int32))
    status()
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_against_each_alone(cuda, dtype):
    c, rel, w, _ = case("mixed")
    ids = np.random.default_rng(6).integers(0, c["vocab"], (5, 66))
    qs = [Sequence(c, w, r, trials=3) for r in ids]
    m = build(c, rel, w, dtype, max_seq_len=100)
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding(cuda, dtype):
    """Hundreds of single tokens, past every edge of the bias tables and of the key tiles."""
    c, rel, w, _ = case("mixed")
    if "long" not in _cache:
        _cache["long"] = Sequence(c, w, np.random.default_rng(7).integers(0, c["vocab"], 420), trials=2)
    q = _cache["long"]
    m = build(c, rel, w, dtype, max_seq_len=420)
    q.check(run(m, q.ids, [5] + [1] * 415), dtype)
    m.close()


@pytest.mark.parametrize("dtype", DTYPES)
def test_far_key(cuda, dtype):
    """A token is found again over a thousand positions: its query and key point the same way, everything else gets almost no weight."""
    c, rel = config(40, 64, [(attention(4, 2, 64, 16, 8, 30, scale=1.0), None), (mamba(32, 8, 4, 2), dense(32))])
    w = weights(c, rel, seed=3)
    rng = np.random.default_rng(3)
    mark, ask, fill = 1, 2, 3
    e, d = (np.linalg.qr(rng.standard_normal((64, 3)))[0].T for _ in range(2))      # three directions of the stream, three of queries and keys
    for row, v in ((mark, e[0]), (ask, e[1]), (fill, e[2])):
        w["embed"][row] = 8 * v
    k, qw = np.outer(d[0], e[0]) + np.outer(d[1], e[1] + e[2]), np.outer(d[0], e[1]) + np.outer(d[2], e[0] + e[2])
    w["l0.mix.k"], w["l0.mix.q"] = np.concatenate([k] * 2), np.concatenate([qw] * 4)
    w["l0.mix.pb"] = np.full(4, -40.0)
    w["l0.mix.rel"] *= 0.1
    w["l0.mix.talk"] = np.eye(4) + 0.05 * rng.standard_normal((4, 4))
    from helpers import bf16_round
    w = {k: bf16_round(np.asarray(v, np.float32)).reshape(np.shape(v)) for k, v in w.items()}
    ids = np.full(1400, fill)
    ids[70], ids[1300], ids[-1] = mark, ask, ask
    q = Sequence(c, w, ids, trials=2)
    without = ids.copy()
    without[70] = fill
    other = reference(c, w).forward(without)
    for at in (1300, 1399):
        assert errors(q.want[at:at + 1], other[at:at + 1])[0] > 0.2
    m = build(c, rel, w, dtype, max_seq_len=1400)
    for cuts in ([1400], [71, 1229, 99, 1], [1290] + [1] * 12 + [97, 1]):
        got = run(m, ids, cuts)
        for at in (1300, 1399):
            q.check(got[at:at + 1], dtype, at)
    m.close()


@pytest.mark.parametrize("use_graph", [True, False])
@pytest.mark.parametrize("name,dtype", [("mixed", "bfloat16"), ("ragged", "bfloat16"), ("mixed", "float32"), ("recurrent", "float32"), ("wide", "bfloat16")])
def test_greedy_generation(cuda, name, dtype, use_graph):
    """Generator on a batch of prompts: every token an arg-max of the reference's logits for the same history."""
    c, rel, w, q = case(name)
    B, P, n = 3, 37, 40
    prompt = np.random.default_rng(8).integers(0, c["vocab"], (B, P)).astype(np.int32)
    m = build(c, rel, w, dtype, max_seq_len=80)
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


def test_model_folder_and_errors(cuda, tmp_path):
    from vesper_b200.model import load_model
    c, rel, w, q = case("mixed")
    save(tmp_path, c, w)
    m = load_model(str(tmp_path), "float32", max_seq_len=160)
    q.check(run(m, q.ids[:50], [50]), "float32")
    m.close()
    save(tmp_path, c, {k: v for k, v in w.items() if k != "l1.mlp.e3.down"})
    with pytest.raises(RuntimeError, match="l1.mlp.e3.down"):
        load_model(str(tmp_path))
    for name, bad in (("l0.mix.rel", w["l0.mix.rel"][:, :-1]), ("head", w["head"][:-1]), ("l2.mix.vmix", w["l2.mix.vmix"].reshape(1))):
        save(tmp_path, c, dict(w, **{name: bad}))
        with pytest.raises(RuntimeError, match=name):
            load_model(str(tmp_path))


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_replay(cuda, tmp_path, dtype):
    c, rel, w, q = case("ragged")
    save(tmp_path, c, w)
    ids, other = q.ids, np.random.default_rng(9).integers(0, c["vocab"], 25)
    q2 = Sequence(c, w, other)
    steps = [dict(entries=[dict(id="a", tokens=ids[:60].tolist(), want=[0, 59, 7])], end=[]),
             dict(entries=[dict(id="b", tokens=other[:2].tolist(), want=[])], end=[]),
             dict(entries=[dict(id="a", tokens=ids[60:61].tolist(), want=[0])], end=["a"]),
             dict(entries=[dict(id="b", tokens=other[2:].tolist(), want=[22, 1])], end=["b"]),
             dict(entries=[dict(id="a", tokens=ids[:3].tolist(), want=[2])], end=["a"])]
    text = "".join(json.dumps(dict(s, step=i)) + "\n" for i, s in enumerate(steps))
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "100"],
                       input=text, capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert r.stdout.split("\n")[:5] == [f"done {i}" for i in range(5)]
    rows = {0: [(q, 0), (q, 59), (q, 7)], 2: [(q, 60)], 3: [(q2, 24), (q2, 3)], 4: [(q, 2)]}
    assert not (tmp_path / "1.f32").exists()
    for i, x in rows.items():
        got = np.fromfile(tmp_path / f"{i}.f32", "<f4").reshape(len(x), c["vocab"])
        for y, (seq, at) in zip(got, x):
            seq.check(y[None], dtype, at)


def test_generate_command(cuda, tmp_path):
    c, rel, w, _ = case("mixed")
    save(tmp_path, c, w)
    r = subprocess.run([sys.executable, "-m", "vesper_b200.generate", "--model", str(tmp_path), "--new", "6", "--prompt", "5 9 2", "--prompt", "1 1 7"],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    lines = [[int(t) for t in line.split()] for line in r.stdout.strip().splitlines()]
    m = build(c, rel, w, "bfloat16", max_seq_len=100)
    assert np.array_equal(m.generate_greedy(np.array([[5, 9, 2], [1, 1, 7]]), 6)[0], np.array(lines))
    m.close()
