"""Zudisun decoders without a GPU: the plain model's own consistency, its mechanisms by hand, configuration errors, workspace plans."""
import copy
import ctypes as C
import math

import numpy as np
import pytest

import zudisun_reference as ref
from zudisun_cases import CASES, reference, weights


@pytest.mark.parametrize("name", sorted(CASES))
def test_reference_does_not_depend_on_portions(name):
    c, rel = CASES[name]
    w = weights(c, rel, seed=1)
    ids = np.random.default_rng(0).integers(0, c["vocab"], 40)
    whole = reference(c, w).forward(ids)
    r = reference(c, w)
    parts, at = [], 0
    for n in (1, 2, 20, 1, 3, 1, 12):
        parts.append(r.forward(ids[at:at + n]))
        at += n
    assert np.abs(np.concatenate(parts) - whole).max() <= 1e-9 * np.abs(whole).max()


def test_distance_buckets():
    b = [ref.distance_bucket(n, 8, 64) for n in range(100)]
    # a row each up to 3, then quarters of the logarithm from 4 to 64: edges at 8, 16, 32
    assert b[:4] == [0, 1, 2, 3] and b[4] == 4 and b[7] == 4 and b[8] == 5 and b[15] == 5 and b[16] == 6 and b[31] == 6 and b[32] == 7 and b[99] == 7
    assert [ref.distance_bucket(n, 2, 5) for n in range(4)] == [0, 1, 1, 1]
    assert max(ref.distance_bucket(n, 32, 200) for n in range(1000)) == 31 and ref.distance_bucket(199, 32, 200) == 31


def test_mechanisms_by_hand():
    assert ref.query_temperature(0, 0.5, 4) == 1.0 and ref.query_temperature(2, 0.5, 4) == 1.0
    assert np.isclose(ref.query_temperature(3, 0.5, 4), 1 + 0.5 * math.log(2)) and np.isclose(ref.query_temperature(11, 0.5, 4), 1 + 0.5 * math.log(4))
    # two heads on one key head: mixed scores, bias by distance, an offset per head, weights that do not add up to one
    q, k, v = np.array([[[1.0], [2.0]]]), np.array([[[3.0]], [[5.0]]]), np.array([[[10.0]], [[100.0]]])
    rel, talk, pb = np.array([[0.1, 0.2], [0.3, 0.4]]), np.array([[1.0, 0.5], [0.0, 2.0]]), np.array([-1.0, -2.0])
    o = ref.sigmoid_attention(q, k, v, [1], 0.5, rel, 2, talk, pb)
    s0 = [1.5 + 0.3, 3.0 + 0.4]                        # key 0, distance 1, both heads
    s1 = [2.5 + 0.1, 5.0 + 0.2]
    sg = lambda z: 1 / (1 + math.exp(-z))
    assert np.isclose(o[0, 0, 0], 10 * sg(s0[0] + 0.5 * s0[1] - 1) + 100 * sg(s1[0] + 0.5 * s1[1] - 1))
    assert np.isclose(o[0, 1, 0], 10 * sg(2 * s0[1] - 2) + 100 * sg(2 * s1[1] - 2))
    # the state after one token is dt x B; a second token with x = 0 decays it per channel and state
    y, S = ref.selective_scan(np.array([[2.0], [0.0]]), np.array([[0.5], [2.0]]), np.log(np.array([[1.0, 3.0]])), np.array([[3.0, 1.0], [7.0, 7.0]]), np.ones((2, 2)), np.array([10.0]),
                              np.zeros((1, 2)))
    assert np.allclose(y[:, 0], [3 + 1 + 20, 3 * math.exp(-2) + math.exp(-6)]) and np.allclose(S, [[3 * math.exp(-2), math.exp(-6)]])


def test_routing_by_hand():
    z = np.array([3.0, -3.0, 1.0, 0.9, 2.0, -5.0])
    s = 1 / (1 + np.exp(-z))
    ids, w = ref.route(z, np.zeros(6), 2, 3, 1, 2.0)   # group sums: experts 2 and 3 together beat 0 and 1, and 4 and 5
    assert ids.tolist() == [2, 3] and np.allclose(w, 2 * s[[2, 3]] / (s[2] + s[3]))
    ids, _ = ref.route(z, np.zeros(6), 2, None, None, 1.0)
    assert ids.tolist() == [0, 4]
    ids, w = ref.route(z, np.array([-9, 0, 0, 0, 0, 0.5]), 3, 3, 2, 1.0)        # the correction moves the choice, not the weights
    assert ids.tolist() == [4, 2, 3] and np.allclose(w, s[ids] / s[ids].sum())
    ids, _ = ref.route(z, np.full(6, -20.0), 4, 3, 2, 1.0)                      # all negative: the third group stays out
    assert set(ids.tolist()) == {0, 1, 2, 3}


def _changed(name, layer, path, value):
    c = copy.deepcopy(CASES[name][0])
    at = c["layers"][layer]
    for k in path[:-1]:
        at = at[k]
    at[path[-1]] = value
    return c


@pytest.mark.parametrize("c,text", [
    (_changed("mixed", 0, ["mlp", "kind"], "tree"), "no feed-forward of kind"),
    (_changed("mixed", 0, ["type"], "rwkv"), "no sequence mixer of type"),
    (_changed("mixed", 0, ["mixer", "kv_heads"], 4), "divisible by kv_heads"),
    (_changed("mixed", 0, ["mixer", "q_temp"], dict(coef=1.0)), "missing key 'every'"),
    (_changed("mixed", 1, ["mixer", "state"], 0), "'state' must be positive"),
    (_changed("mixed", 1, ["mlp", "router", "groups"], dict(count=4, keep=1)), "divide into the groups"),
    (_changed("mixed", 1, ["mlp", "router", "groups"], dict(count=6, keep=1)), "hold 'top' experts"),
    (_changed("mixed", 2, ["mlp", "router", "top"], 13), "'top' exceeds"),
    (_changed("mixed", 2, ["mixer", "vdim"], 16), "one number of value columns"),
    (dict(CASES["mixed"][0], loop=dict(start=0, stop=2, times=2)), "no loop"),
])
def test_configuration_errors(lib, c, text):
    from vesper_b200.build import build_host
    build_host()
    from vesper_b200.model import model_from_config
    with pytest.raises(RuntimeError, match=text):
        model_from_config(c)


def test_workspace_plans(lib):
    """Sizes are refused or planned without a device; struct_size mismatches are refused."""
    from vesper_b200 import hybrid_capi as hc
    L = hc.load()
    a = hc.SigattnArgs(struct_size=C.sizeof(hc.SigattnArgs), dtype=1, B=2, T=1, H=16, G=4, dim=128, vdim=128, cap=4096, n_bias=5)
    sizes = []
    for n in (1, 64, 65, 1000, 4096, 100000, 0):
        a.max_len = n
        sizes.append(L.vb200_sigattn_workspace_bytes(C.byref(a)))
    assert sizes == sorted(sizes) and sizes[-1] == sizes[-2] == sizes[-3] and sizes[0] < sizes[2]
    assert sizes[0] == 2 * 16 * 512 * 2 + 2 * 16 * 128 * 4                  # mixed queries in bf16, one partial sum per head
    a.H = 15
    assert L.vb200_sigattn_workspace_bytes(C.byref(a)) == 0
    m = hc.MoeArgs(struct_size=C.sizeof(hc.MoeArgs), dtype=1, M=512, dim=64, ff=32, ff_shared=32, experts=8, top=2, groups=4, keep=1)
    assert L.vb200_moe_rows(C.byref(m)) == 2                                 # a prompt leaves its experts' rows to the norm
    m.M = 1
    assert L.vb200_moe_rows(C.byref(m)) == 0 and L.vb200_moe_workspace_bytes(C.byref(m)) > 0
    for change in (dict(top=3), dict(groups=3), dict(keep=5), dict(experts=0), dict(struct_size=8)):
        b = hc.MoeArgs.from_buffer_copy(m)
        for k, v in change.items():
            setattr(b, k, v)
        assert L.vb200_moe_workspace_bytes(C.byref(b)) == 0 and L.vb200_moe_forward(C.byref(b)) == -1, change
    s = hc.SelectiveArgs(struct_size=C.sizeof(hc.SelectiveArgs), dtype=1, B=1, T=1, inner=512, N=16, rank=32, taps=4)
    assert L.vb200_selective_workspace_bytes(C.byref(s)) == 512 * 2 + 256    # convolution output, step sizes and B and C before the scan
    s.inner = 500
    assert L.vb200_selective_forward(C.byref(s)) == -3
    n = hc.NormAddArgs(struct_size=4)
    assert L.vb200_norm_add(C.byref(n)) == -1 and L.vb200_selective_forward(None) == -1
