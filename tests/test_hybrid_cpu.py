"""Hybrid decoders without a GPU: the plain model's own consistency, configuration errors, workspace plans."""
import ctypes as C
import json

import numpy as np
import pytest

import hybrid_reference as ref
from hybrid_cases import CASES, reference, weights


@pytest.mark.parametrize("name", sorted(CASES))
def test_reference_does_not_depend_on_portions(name):
    c = CASES[name]
    w = weights(c, seed=1)
    ids = np.random.default_rng(0).integers(0, c["vocab"], 60)
    whole = reference(c, w).forward(ids)
    r = reference(c, w)
    parts, at = [], 0
    for n in (1, 2, 30, 1, 3, 1, 22):
        parts.append(r.forward(ids[at:at + n]))
        at += n
    assert np.abs(np.concatenate(parts) - whole).max() <= 1e-9 * np.abs(whole).max()


def test_reference_mechanisms():
    rng = np.random.default_rng(1)
    # rotation depends on position differences only
    q, k = rng.standard_normal((2, 1, 8))
    dots = [float(ref.rotate_half(q, [p + 5], 100.0)[0] @ ref.rotate_half(k, [p], 100.0)[0]) for p in (0, 3, 1000)]
    assert np.allclose(dots, dots[0])
    # window and sink by hand: query 2 sees keys 1 and 2 of equal score, and a sink of score 0
    v = np.array([1.0, 2.0, 4.0]).reshape(3, 1, 1)
    o = ref.window_attention_with_sink(np.zeros((1, 1, 1)), np.zeros((3, 1, 1)), v, [2], [0, 1, 2], 1.0, 2, np.zeros(1))
    assert np.isclose(o[0, 0, 0], (2.0 + 4.0) / 3.0)
    # the state after one token is dt B x^T, and decays by exp(-exp(A_log) dt)
    x, B, dt = np.array([[[2.0]], [[0.0]]]), np.array([[[3.0]], [[1.0]]]), np.array([[0.5], [2.0]])
    y, S = ref.ssd_scan(x, B, np.ones((2, 1, 1)), dt, np.zeros(1), np.zeros(1), np.zeros((1, 1, 1)))
    assert np.allclose(y[:, 0, 0], [3.0, 3.0 * np.exp(-2.0)]) and np.allclose(S, 3.0 * np.exp(-2.0))
    out, before = ref.causal_conv(np.array([[1.0], [2.0]]), np.array([[7.0], [5.0]]), np.array([[100.0, 10.0, 1.0]]), np.array([0.5]))
    assert out[:, 0].tolist() == [751.5, 512.5] and before[:, 0].tolist() == [1.0, 2.0]
    assert ref.bigram_rows([4, 5], None, 10, 3, 2).tolist() == [10, 2] and ref.bigram_rows([4], 5, 10, 3, 2).tolist() == [3]


@pytest.mark.parametrize("change,text", [
    (dict(architecture="Unheard"), "no model class"),
    (dict(layers=[dict(type="latent_attention", mixer={}, mlp=dict(kind="gated", ff=8))]), "no feed-forward of kind"),
    (dict(loop=dict(start=1, stop=1, times=2)), "loop"),
    (dict(loop=dict(start=0, stop=9, times=2)), "loop"),
    (dict(norm={}), "missing key 'eps'"),
    (dict(width=0), "positive"),
])
def test_configuration_errors(lib, change, text):
    from vesper_b200.build import build_host
    build_host()
    from vesper_b200.model import model_from_config
    with pytest.raises(RuntimeError, match=text):
        model_from_config(dict(CASES["tail"], **change))


def test_malformed_json(lib):
    from vesper_b200.build import build_host
    build_host()
    from vesper_b200.model import load_host
    L = load_host()
    for text in ("{", '{"a": 1,}', '{"architecture": nope}', "[1] x", ""):
        assert not L.vbh_model_from_config(text.encode(), 0, 0, 0)
        assert b"JSON" in L.vbh_last_error(), text
    assert json.loads('"\\u00e9"') == "é"


def test_workspace_plans(lib):
    """Decode workspaces grow with the longest length and stop at the ring; struct_size mismatches are refused."""
    from vesper_b200 import hybrid_capi as hc
    L = hc.load()
    a = hc.LatentArgs(struct_size=C.sizeof(hc.LatentArgs), dtype=1, B=2, T=1, H=16, dim=128, rot_dim=64, vdim=128, rank=512, window=4096, ring=4096)
    sizes = []
    for n in (1, 64, 65, 1000, 4096, 100000, 0):
        a.max_len = n
        sizes.append(L.vb200_latent_workspace_bytes(C.byref(a)))
    assert sizes == sorted(sizes) and sizes[-1] == sizes[-2] == sizes[-3] and sizes[0] < sizes[2]
    q = 2 * 16 * 576
    assert sizes[0] == 4 * (q + 2 * 16 * 516)              # one slice: queries and one record per head
    s = hc.SsdArgs(struct_size=C.sizeof(hc.SsdArgs), dtype=1, B=1, T=1, H=8, P=64, N=128, G=1, taps=4, norm_groups=1)
    assert L.vb200_ssd_workspace_bytes(C.byref(s)) == (8 * 64 + 2 * 128) * 2 + 8 * 64 * 4       # convolution output, gated values
    s.struct_size = a.struct_size = 8
    assert L.vb200_ssd_workspace_bytes(C.byref(s)) == 0 and L.vb200_latent_workspace_bytes(C.byref(a)) == 0
    assert L.vb200_ssd_forward(C.byref(s)) == -1 and L.vb200_latent_decode(C.byref(a)) == -1 and L.vb200_embed_sequence(None) == -1
