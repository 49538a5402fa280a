"""The operators behind Zudisun decoders (include/vesper_b200_hybrid.h) on the GPU against the plain equations of
zudisun_reference.py, one mechanism at a time.

Tolerances: fp32 forms 2e-5 of the largest output; bf16 forms 1.2e-2 (values are rounded to bf16 between steps on both sides)."""
import numpy as np
import pytest

import zudisun_reference as ref
from helpers import bf16_round
from hybrid_reference import causal_conv, rms_norm, silu, softplus

pytestmark = pytest.mark.gpu

TOL = {"f32": 2e-5, "bf16": 1.2e-2}


def _torch(x, cuda, dtype=None):
    import torch
    t = torch.from_numpy(np.ascontiguousarray(x)).to(cuda)
    return t.to(dtype) if dtype is not None else t


def _f32(x, cuda):
    return _torch(np.asarray(x, np.float32), cuda)


def _np(t):
    return t.detach().double().cpu().numpy()


def _dt(kind):
    import torch
    return torch.float32 if kind == "f32" else torch.bfloat16


def _rnd(kind):
    return (lambda a: a) if kind == "f32" else (lambda a: bf16_round(np.asarray(a, np.float32)).astype(np.float64))


def _close(got, want, tol, what=None):
    err = np.abs(_np(got) - want).max() / max(np.abs(want).max(), 1e-6)
    assert err <= tol, (what, err)


def _status():
    from vesper_b200 import capi
    capi.check_kernel_status(0)


# ---- norms and gated products --------------------------------------------------------------------

@pytest.mark.parametrize("M,dim,count", [(5, 48, 45), (3, 2048, 2048), (2, 9000, 8997)])
def test_norm_of_a_sublayers_output(cuda, M, dim, count):
    import torch
    from vesper_b200 import hybrid_capi as hc
    rng = np.random.default_rng(0)
    x, y = rng.standard_normal((2, M, dim)).astype(np.float32)
    x[:, count:] = y[:, count:] = 0
    w, scale = rng.standard_normal((2, dim)).astype(np.float32)
    xt = _torch(x, cuda)
    copy = hc.norm_add(xt, _torch(y, cuda), _torch(w, cuda), 1e-3, count=count, scale=_torch(scale, cuda), copy=True)
    norm = lambda v: v / np.sqrt((v * v).sum(-1, keepdims=True) / count + 1e-3) * w
    want = x.astype(np.float64) + norm(y.astype(np.float64))
    _close(xt, want, 1e-6)
    _close(copy, want * scale, 2 ** -8)
    assert (_np(xt)[:, count:] == 0).all()
    # rows left by the experts are added ahead of the norm; the copy without a scale
    rows, gather = bf16_round(rng.standard_normal((M * 3, dim))), rng.permutation(M * 3).reshape(M, 3).astype(np.int32)
    rows[:, count:] = 0
    for first in (y, None):
        xt = _torch(x, cuda)
        copy = hc.norm_add(xt, None if first is None else _torch(first, cuda), _torch(w, cuda), 1e-3, count=count, rows=_torch(rows, cuda, torch.bfloat16),
                           gather=_torch(gather, cuda), copy=True)
        want = x + norm((0 if first is None else first.astype(np.float64)) + rows.astype(np.float64)[gather].sum(1))
        _close(xt, want, 1e-6)
        _close(copy, want, 2 ** -8)
    _status()


@pytest.mark.parametrize("M", [1, 16, 40, 64, 65, 300])
@pytest.mark.parametrize("N,K", [(72, 64), (300, 136)])
def test_relu_gate_with_bias(cuda, M, N, K):
    import torch
    from vesper_b200 import capi, hybrid_capi as hc
    rng = np.random.default_rng(M)
    x, w, b = bf16_round(rng.standard_normal((M, K))), bf16_round(rng.standard_normal((2 * N, K)) / np.sqrt(K)), rng.standard_normal(2 * N).astype(np.float32)
    z = x.astype(np.float64) @ w.T.astype(np.float64) + b
    want = np.maximum(z[:, ::2], 0) * z[:, 1::2]
    ld = (N + 7) // 8 * 8
    out = torch.full((M, ld), 7.0, dtype=torch.bfloat16, device=cuda)
    xb, wb, bt, xf, wf = _torch(x, cuda, torch.bfloat16), _torch(w, cuda, torch.bfloat16), _torch(b, cuda), _f32(x, cuda), _f32(w, cuda)
    capi.check(hc.load().vb200_linear_bias(0, hc._stream(), xb.data_ptr(), K, wb.data_ptr(), K, bt.data_ptr(), out.data_ptr(), ld, M, 2 * N, K, 5, 0))
    _close(out[:, :N], want, 2 ** -7)
    assert (out[:, N:] == 7.0).all()
    for epi, act in ((5, lambda g: np.maximum(g, 0)), (3, silu)):
        f = torch.empty(M, N, device=cuda)
        capi.check(hc.load().vb200_linear_f32_ex(0, hc._stream(), xf.data_ptr(), K, wf.data_ptr(), K, bt.data_ptr(), None, f.data_ptr(), N, M, 2 * N, K, epi))
        _close(f, act(z[:, ::2]) * z[:, 1::2], 1e-5)
    _status()


# ---- sigmoid attention ---------------------------------------------------------------------------

SIG = {  # H, G, dim, vdim, scale, temp (coef, every), distances
    "small": (8, 2, 32, 16, 0.3, (0.4, 16), 40),
    "one head each": (4, 4, 24, 40, 0.2, (0.7, 5), 9),
    "odd sizes": (6, 3, 10, 12, 0.4, None, 130),
    "odd values": (6, 2, 16, 20, 0.3, (0.3, 7), 20),
    "widest": (16, 4, 128, 128, 0.05, (0.5, 32), 70),
    "many heads": (20, 2, 64, 72, 0.1, (0.2, 3), 25),
    "one head": (1, 1, 8, 8, 0.9, (0.5, 64), 1),
    "group of ten": (10, 1, 48, 200, 0.1, None, 33),
    "large rows": (12, 12, 64, 64, 0.1, (0.1, 9), 30),
    "pairs of heads": (12, 6, 40, 64, 0.15, (0.3, 50), 140),
    "pairs, wide values": (8, 2, 104, 128, 0.08, None, 300),
}


class SigCase:
    """One sequence: projections, the plain result, and a core to run them through.  One key per sequence stands out for later queries."""

    def __init__(self, name, kind, L, seed=0, slots=1, cap=None):
        self.H, self.G, self.dim, self.vdim, self.scale, self.temp, nb = SIG[name]
        self.name, self.kind, self.L, self.cap = name, kind, L, cap or L
        self.slots = slots
        rng = self.rng = np.random.default_rng(seed)
        H = self.H
        self.talk = (np.eye(H) + rng.standard_normal((H, H)) * 0.3 / np.sqrt(H)).astype(np.float32)
        self.bias = (rng.standard_normal((H, nb)) * 1.5 - 4.0).astype(np.float32)
        self.lam = 0.35

    def sequence(self, L=None):
        L, rng, H, G, d, dv = L or self.L, self.rng, self.H, self.G, self.dim, self.vdim
        q, k, v, g = (rng.standard_normal((L, n, m)) for n, m in ((H, d), (G, d), (G, dv), (H, 1)))
        # every few positions a query looks for one earlier key, whose value is large: a wrong key, distance or split shows
        for i in range(3, L, 4):
            j = int(rng.integers(0, i))
            q[i] = 0.3 * q[i] + 3.0 * np.repeat(k[j], H // G, axis=0)
            v[j] *= 3.0
        return _rnd(self.kind)(np.concatenate([a.reshape(L, -1) for a in (q, k, v, g)], axis=1))

    def core(self, cuda):
        from vesper_b200 import hybrid_capi as hc
        t = self.temp or (0.0, 0)
        return hc.SigmoidCore(H=self.H, G=self.G, dim=self.dim, vdim=self.vdim, scale=self.scale, eps=1e-5, talk=_torch(self.talk, cuda), bias=_torch(self.bias, cuda),
                              slots=self.slots, cap=self.cap, dtype=_dt(self.kind), temp_coef=t[0], temp_every=t[1])

    def want(self, p, first=None):
        """Plain result [L, H * vdim] of projections [L, cols] of a whole sequence; first: values of the first mixing layer."""
        H, G, d, dv, L, rnd = self.H, self.G, self.dim, self.vdim, len(p), _rnd(self.kind)
        q, k, v, g = np.split(p, [H * d, (H + G) * d, (H + G) * d + G * dv], axis=1)
        q, k = rms_norm(q.reshape(L, H, d), 1e-5), rnd(rms_norm(k.reshape(L, G, d), 1e-5))
        if self.temp:
            q = q * np.array([ref.query_temperature(i, *self.temp) for i in range(L)])[:, None, None]
        if first is not None:
            v = rnd((1 - self.lam) * v + self.lam * first)
        # the bias is given per distance, mixed already: a table with a row per distance, taken through the inverse of the mixing
        nb = self.bias.shape[1]
        out = np.zeros((L, H, dv))
        v = v.reshape(L, G, dv)
        for t in range(L):
            s = np.stack([(k[:t + 1, h // (H // G)] @ q[t, h]) * self.scale for h in range(H)])
            w = ref.sigmoid(self.talk.astype(np.float64) @ s + self.bias.astype(np.float64)[:, np.minimum(t - np.arange(t + 1), nb - 1)])
            for h in range(H):
                out[t, h] = w[h] @ v[:t + 1, h // (H // G)]
        return (out * ref.sigmoid(g)[:, :, None]).reshape(L, H * dv)

    def run(self, core, cuda, p, cuts, slot=0, form=0, **kw):
        import torch
        out, at = [], 0
        slots = torch.full((1,), slot, dtype=torch.int32, device=cuda)
        for n in cuts:
            buf = core.proj_buffer(n)
            buf[:, :p.shape[1]] = _torch(p[at:at + n], cuda, self.dtype_of(core))
            out.append(_np(core.forward(buf, 1, at, slots=slots, form=form, max_len=at + n, **kw)))
            at += n
        _status()
        return np.concatenate(out)

    @staticmethod
    def dtype_of(core):
        return core.dtype


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(SIG))
def test_sigmoid_attention_prompts_portions_and_tokens(cuda, name, kind):
    L = 300
    c = SigCase(name, kind, L, seed=len(name), slots=3)
    p = c.sequence()
    want = c.want(p)
    core = c.core(cuda)
    scale = np.abs(want).max()
    # position-wise: early positions have few keys and small outputs
    close = lambda got, w, tag: np.testing.assert_array_less(np.abs(got - w).max(-1), TOL[kind] * np.maximum(np.abs(w).max(-1), 0.25 * scale), err_msg=f"{name} {tag}")
    close(c.run(core, cuda, p, [L]), want, "prompt")
    tuned_prompt = core.last_kernel()
    close(c.run(core, cuda, p, [129, 2, 3, 64, 1, 60, L - 259], slot=2), want, "portions")
    close(c.run(core, cuda, p, [L - 40] + [1] * 40, slot=1), want, "decoded")
    tuned_step = core.last_kernel()
    close(c.run(core, cuda, p[:50], [1] * 50, slot=1), want[:50], "from the first token, in a used slot")
    if kind == "bf16":
        fits = c.G * c.dim <= 512 and c.vdim % 8 == 0
        pair = fits and (c.H // c.G) % 2 == 0 and c.vdim in (64, 128) and c.G * c.dim >= 192
        assert tuned_prompt == ("sig_prefill_sm100_kernel (pair)" if pair else "sig_prefill_sm100_kernel" if fits else "sig_attend_generic_kernel")
        if pair:
            close(c.run(core, cuda, p, [L], form=2), want, "single SMs")
            close(c.run(core, cuda, p, [129, L - 129], form=2), want, "single SMs, portions")
        assert (tuned_step == "sig_decode_mma_kernel") == (fits and c.G * c.vdim <= 512)
        close(c.run(core, cuda, p, [L - 3, 1, 1, 1], form=1), want, "CUDA cores")


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_sigmoid_attention_batches_in_permuted_slots(cuda, kind):
    import torch
    B, L = 3, 90
    c = SigCase("small", kind, L, seed=3, slots=5, cap=100)
    ps = [c.sequence() for _ in range(B)]
    wants = [c.want(p) for p in ps]
    core = c.core(cuda)
    core.k_cache.normal_(); core.v_cache.normal_()                    # what earlier sequences left
    slots = _torch(np.array([4, 1, 3], np.int32), cuda)
    keep = core.v_cache[[0, 2]].clone()
    at = 0
    for n in (70, 1, 2, 1, 1, 15):
        buf = core.proj_buffer(B * n)
        buf[:, :ps[0].shape[1]] = _torch(np.concatenate([p[at:at + n] for p in ps]), cuda, core.dtype)
        y = _np(core.forward(buf, B, at, slots=slots)).reshape(B, n, -1)
        for b in range(B):
            assert np.abs(y[b] - wants[b][at:at + n]).max() <= TOL[kind] * np.abs(wants[b]).max(), (n, at, b)
        at += n
    assert torch.equal(core.v_cache[[0, 2]], keep)
    # decoding at unequal lengths: rows of one call stand at positions of their own
    core2 = c.core(cuda)
    lens = [60, 7, 31]
    for b in range(B):
        c.run(core2, cuda, ps[b], [lens[b]], slot=int(slots[b]))
    for step in range(4):
        buf = core2.proj_buffer(B)
        buf[:, :ps[0].shape[1]] = _torch(np.stack([ps[b][lens[b] + step] for b in range(B)]), cuda, core2.dtype)
        y = _np(core2.forward(buf, B, 0, pos=_torch(np.array([n + step for n in lens], np.int32), cuda), slots=slots, max_len=100))
        for b in range(B):
            w = wants[b][lens[b] + step]
            assert np.abs(y[b] - w).max() <= TOL[kind] * np.abs(wants[b]).max(), (step, b)
    _status()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_values_mixed_with_the_first_layers(cuda, kind):
    import torch
    L = 40
    c = SigCase("small", kind, L, seed=7)
    p1, p2 = c.sequence(), c.sequence()
    vcols = slice((c.H + c.G) * c.dim, (c.H + c.G) * c.dim + c.G * c.vdim)
    first, second = c.core(cuda), c.core(cuda)
    want1, want2 = c.want(p1), c.want(p2, first=p1[:, vcols])
    assert np.abs(want2 - c.want(p2)).max() > 0.1 * np.abs(want2).max()
    at = 0
    for n in (25, 1, 1, 2, 11):
        values = torch.full((n, c.G * c.vdim), float("nan"), device=cuda, dtype=first.dtype)
        for core, p, want, role in ((first, p1, want1, 1), (second, p2, want2, 2)):
            buf = core.proj_buffer(n)
            buf[:, :p.shape[1]] = _torch(p[at:at + n], cuda, core.dtype)
            y = core.forward(buf, 1, at, value_role=role, lam=c.lam, first_values=values)
            _close(y, want[at:at + n], TOL[kind] * np.abs(want).max() / np.abs(want[at:at + n]).max())
        at += n
    _status()


def test_sigmoid_attention_far_key_and_bias_edges(cuda):
    """One key among two thousand, and a bias that differs in one distance only: both show in the output, in prompts and in decoding."""
    L, kind = 2050, "bf16"
    c = SigCase("small", kind, L, seed=9)
    c.temp = None
    c.bias[:] = -12.0
    p = 0.05 * c.rng.standard_normal((L, c.H * (c.dim + 1) + c.G * (c.dim + c.vdim)))
    H, G, d, dv = c.H, c.G, c.dim, c.vdim
    k = p[:, H * d:(H + G) * d].reshape(L, G, d)
    q = p[:, :H * d].reshape(L, H, d)
    v = p[:, (H + G) * d:(H + G) * d + G * dv].reshape(L, G, dv)
    v[:] = 0.0
    for far in (0, 1, 127, 128, 1000):                 # keys that the last queries look for, at tile borders
        k[far] = c.rng.standard_normal((G, d))
        v[far] = 1.0 + far / 500
    for i, far in ((L - 1, 0), (L - 2, 1), (L - 3, 127), (L - 4, 128), (L - 5, 1000), (200, 128)):
        q[i] = np.repeat(k[far], H // G, axis=0)
    p = _rnd(kind)(p)
    c.talk = np.eye(H, dtype=np.float32)
    c.scale = 0.6
    rows = [200, L - 5, L - 4, L - 3, L - 2, L - 1]
    want = c.want(p)
    for i in rows:
        assert np.abs(want[i]).max() > 0.2             # the key stands out
    core = c.core(cuda)
    for cuts in ([L], [L - 5] + [1] * 5, [1000, 1045, 2, 3]):
        got = c.run(core, cuda, p, cuts)
        for i in rows:
            assert np.abs(got[i] - want[i]).max() <= 1.5e-2 * np.abs(want[i]).max(), (cuts[:2], i)
    # one distance at a time: its keys get weight, all others none
    nb = c.bias.shape[1]
    v[:] = c.rng.standard_normal(v.shape)
    p[:, (H + G) * d:(H + G) * d + G * dv] = _rnd(kind)(v.reshape(L, -1))
    p[:, :H * d] = 0.0
    p = _rnd(kind)(p)[:200]
    for n in (0, 1, nb - 2, nb - 1):
        c.bias[:] = -30.0
        c.bias[:, n] = 2.0
        core = c.core(cuda)
        want = c.want(p)
        for cuts in ([200], [150] + [1] * 50, [130, 70]):
            got = c.run(core, cuda, p, cuts)
            assert np.abs(got - want).max() <= 1.2e-2 * np.abs(want).max(), (n, cuts[:2])
    _status()


def test_sigmoid_attention_reports_a_full_cache(cuda):
    from vesper_b200 import capi
    c = SigCase("small", "bf16", 8, cap=8)
    core = c.core(cuda)
    p = c.sequence(9)
    c.run(core, cuda, p, [8])
    with pytest.raises(Exception, match="full"):
        c.run(core, cuda, p[:1], [1])                  # fits: position 0 of a new sequence
        buf = core.proj_buffer(1)
        buf[:, :p.shape[1]] = _torch(p[8:9], cuda, core.dtype)
        core.forward(buf, 1, 8, max_len=8)
        capi.check_kernel_status(0)


# ---- selective state-space mixer -----------------------------------------------------------------

SCAN = {  # inner, N, rank, taps
    "small": (40, 24, 16, 4), "two taps": (16, 8, 8, 2), "one tap": (24, 32, 8, 1), "wide state": (24, 128, 8, 3), "wider state": (16, 256, 24, 5), "widest state": (8, 304, 8, 4),
    "many channels": (520, 16, 40, 4), "long rank": (64, 64, 136, 4),
}


def _scan_case(name, kind, cuda, slots, seed=0):
    from vesper_b200 import hybrid_capi as hc
    inner, N, rank, taps = SCAN[name]
    rng, rnd = np.random.default_rng(seed), _rnd(kind)
    w = dict(conv_w=rng.standard_normal((inner, taps)) / np.sqrt(taps), conv_b=0.3 * rng.standard_normal(inner), w_x=rnd(rng.standard_normal((rank + 2 * N, inner)) / np.sqrt(inner)),
             w_dt=rnd(rng.standard_normal((inner, rank)) / np.sqrt(rank)), dt_bias=rng.standard_normal(inner) - 2.0, A_log=np.log(rng.uniform(0.01, 8.0, (inner, N))), D=rng.standard_normal(inner))
    w = {k: np.asarray(v, np.float32) for k, v in w.items()}
    f = {k: _torch(v, cuda) for k, v in w.items()}
    core = hc.SelectiveCore(inner=inner, N=N, rank=rank, taps=taps, conv_w=f["conv_w"], conv_b=f["conv_b"], w_x=f["w_x"], w_dt=f["w_dt"], dt_bias=f["dt_bias"],
                            A=-f["A_log"].double().exp().float(), D=f["D"], slots=slots, dtype=_dt(kind))
    return core, {k: v.astype(np.float64) for k, v in w.items()}, rng


def _scan_want(p, w, name, kind):
    inner, N, rank, taps = SCAN[name]
    rnd = _rnd(kind)
    c, _ = causal_conv(p[:, :inner], np.zeros((taps - 1, inner)), w["conv_w"], w["conv_b"])
    c = rnd(silu(c))
    d = rnd(c @ w["w_x"].T)
    dt = softplus(d[:, :rank] @ w["w_dt"].T + w["dt_bias"])
    y, _ = ref.selective_scan(c, dt, w["A_log"], d[:, rank:rank + N], d[:, rank + N:], w["D"], np.zeros((inner, N)))
    return y * silu(p[:, inner:])


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(SCAN))
def test_selective_scan_portions_and_slots(cuda, name, kind):
    import torch
    B, L = 2, 150
    core, w, rng = _scan_case(name, kind, cuda, slots=4)
    inner = SCAN[name][0]
    ps = [_rnd(kind)(rng.standard_normal((L, 2 * inner))) for _ in range(B)]
    wants = [_scan_want(p, w, name, kind) for p in ps]
    core.state.fill_(1e3); core.conv_state.fill_(9.0)                 # what earlier sequences left
    for slots, cuts in (((3, 1), [L]), ((0, 3), [33, 1, 2, 64, 1, 1, 3, 45]), ((1, 2), [L - 30] + [1] * 30), ((2, 0), [1] * 60)):
        st = _torch(np.array(slots, np.int32), cuda)
        at = 0
        for n in cuts:
            proj = _torch(np.concatenate([p[at:at + n] for p in ps]), cuda, core.dtype)
            y = _np(core.forward(proj, B, torch.full((B,), at, dtype=torch.int32, device=cuda), slots=st)).reshape(B, n, inner)
            for b in range(B):
                assert np.abs(y[b] - wants[b][at:at + n]).max() <= (5e-5 if kind == "f32" else 2e-2) * np.abs(wants[b]).max(), (cuts[:3], at, b)
            at += n
    _status()


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_selective_steps_of_many_sequences(cuda, kind):
    """Enough rows for the step sizes to become a product of their own; sequences at unequal lengths, one of them new."""
    import torch
    name, B = "small", 21
    core, w, rng = _scan_case(name, kind, cuda, slots=B)
    inner = SCAN[name][0]
    lens = [int(n) for n in rng.integers(1, 30, B)]
    lens[5] = 0
    ps = [_rnd(kind)(rng.standard_normal((n + 3, 2 * inner))) for n in lens]
    wants = [_scan_want(p, w, name, kind) for p in ps]
    slots = rng.permutation(B).astype(np.int32)
    core.state.fill_(50.0)
    for b in range(B):
        if lens[b]:
            core.forward(_torch(ps[b][:lens[b]], cuda, core.dtype), 1, torch.zeros(1, dtype=torch.int32, device=cuda), slots=_torch(slots[b:b + 1], cuda))
    for step in range(3):
        proj = _torch(np.stack([ps[b][lens[b] + step] for b in range(B)]), cuda, core.dtype)
        y = _np(core.forward(proj, B, _torch(np.array(lens, np.int32) + np.int32(step), cuda), slots=_torch(slots, cuda)))
        for b in range(B):
            assert np.abs(y[b] - wants[b][lens[b] + step]).max() <= (5e-5 if kind == "f32" else 2e-2) * np.abs(wants[b]).max(), (step, b)
    _status()


def test_selective_scan_keeps_a_long_memory(cuda):
    """A slow decay carries an early input over a thousand tokens, in one portion and over decoded tokens."""
    import torch
    name, L = "two taps", 1200
    core, w, rng = _scan_case(name, "f32", cuda, slots=1)
    inner = SCAN[name][0]
    w["A_log"][:] = np.log(1e-3)
    core.w["A"].fill_(-1e-3)
    p = 1e-3 * rng.standard_normal((L, 2 * inner))
    p[3, :inner] = 20.0
    p[:, inner:] = 2.0
    want = _scan_want(p, w, name, "f32")
    assert np.abs(want[-1]).max() > 1e-4 * np.abs(want).max()
    for cuts in ([L], [600] + [1] * 300 + [300]):
        at, out = 0, []
        for n in cuts:
            out.append(_np(core.forward(_f32(p[at:at + n], cuda), 1, torch.full((1,), at, dtype=torch.int32, device=cuda))))
            at += n
        got = np.concatenate(out)
        assert np.abs(got[-1] - want[-1]).max() <= 2e-4 * np.abs(want[-1]).max()
    _status()


# ---- mixture of experts --------------------------------------------------------------------------

@pytest.mark.parametrize("E,top,groups,keep", [(10, 4, 5, 3), (8, 2, 0, 0), (64, 6, 8, 2), (12, 12, 0, 0), (96, 40, 4, 3), (16, 3, 16, 5), (1000, 7, 10, 4), (6, 1, 2, 1), (1, 1, 0, 0)])
def test_router_choice(cuda, E, top, groups, keep):
    from vesper_b200 import hybrid_capi as hc
    rng = np.random.default_rng(E)
    for shift in (0.0, -2.0):                          # all choices negative: experts outside the kept groups still cannot be chosen
        logits, corr = (2 * rng.standard_normal((37, E))).astype(np.float32), (shift + 0.6 * rng.standard_normal(E)).astype(np.float32)
        lt, ct = _torch(logits, cuda), _torch(corr, cuda)
        ids, w = hc.moe_route(lt, ct, top, groups, keep, 1.7)
        ids, w = ids.cpu().numpy(), _np(w)
        for m in range(37):
            want_ids, want_w = ref.route(logits[m].astype(np.float64), corr.astype(np.float64), top, groups, keep, 1.7) if groups != E or E == 1 else _route_single(logits[m], corr, top, keep, 1.7)
            assert ids[m].tolist() == want_ids.tolist(), (shift, m)
            assert np.abs(w[m] - want_w).max() <= 1e-5 * 1.7
    _status()


def _route_single(z, corr, top, keep, scale):
    """Groups of one expert: a group's score is its expert's."""
    s = ref.sigmoid(z.astype(np.float64))
    ids = np.argsort(-(s + corr), kind="stable")[:keep][:top]
    return ids, s[ids] / s[ids].sum() * scale


@pytest.mark.parametrize("kind,form", [("f32", 1), ("bf16", 1), ("bf16", 2), ("bf16", 0)])
@pytest.mark.parametrize("M,dim,ff,shared,E,top,groups,keep", [(37, 64, 40, 56, 8, 3, 4, 2), (1, 72, 24, 0, 6, 2, 0, 0), (300, 136, 200, 72, 5, 2, 0, 0), (150, 64, 33, 21, 16, 4, 2, 1)])
def test_mixture_of_experts(cuda, kind, form, M, dim, ff, shared, E, top, groups, keep):
    import torch
    from vesper_b200 import hybrid_capi as hc
    rng, rnd = np.random.default_rng(M), _rnd(kind)
    r = lambda *s: rnd(rng.standard_normal(s) / np.sqrt(s[-1]))
    x, router, corr = rnd(rng.standard_normal((M, dim))), r(E, dim) * 3, (0.4 * rng.standard_normal(E)).astype(np.float32)
    gate, up, down = r(E, ff, dim), r(E, ff, dim), r(E, dim, ff)
    sh = (r(shared, dim), r(shared, dim), r(dim, shared)) if shared else None
    router = rnd(router)
    core = hc.MoeCore(router=_f32(router, cuda), correction=_torch(corr, cuda), gate=_f32(gate, cuda), up=_f32(up, cuda), down=_f32(down, cuda),
                      shared=tuple(_f32(a, cuda) for a in sh) if sh else None, top=top, groups=groups, keep=keep, scale=2.2, dtype=_dt(kind))
    y, rows, gather = core.forward(_torch(x, cuda, core.dtype), form=form)
    torch.cuda.synchronize()
    got = _np(y)
    if form == 2:
        assert rows is not None and core.last_kernel().startswith("linear_wide_kernel")
    if rows is not None:
        assert sorted(gather.flatten().tolist()) == list(range(M * top))
        got = got + _np(rows)[gather.cpu().numpy()].sum(1)
    f = lambda v, g, u, d: rnd(silu(g @ v) * (u @ v)) @ d.T
    want, logits, close_call = np.zeros((M, dim)), x @ router.T, np.zeros(M, bool)
    for m in range(M):
        ids, w = ref.route(logits[m], corr.astype(np.float64), top, groups, keep, 2.2)
        want[m] = sum(we * f(x[m], gate[e], up[e], down[e]) for e, we in zip(ids, w))
        if sh:
            want[m] += f(x[m], *sh)
        close_call[m] = set(ids) != set(ref.route(logits[m] + 1e-4 * rng.standard_normal(E), corr.astype(np.float64), top, groups, keep, 2.2)[0])
    assert close_call.mean() < 0.2
    err = np.abs(got - want).max(-1)[~close_call].max() / np.abs(want).max()
    assert err <= TOL[kind], err
    _status()


def test_experts_without_tokens(cuda):
    """Every token of a prompt chooses the same expert, the last one: all other groups of the sorted rows are empty."""
    import torch
    from vesper_b200 import hybrid_capi as hc
    rng = np.random.default_rng(4)
    E, dim, ff, M = 7, 64, 64, 300
    x = bf16_round(rng.standard_normal((M, dim)))
    gate, up, down = (bf16_round(rng.standard_normal(s) / 8) for s in ((E, ff, dim), (E, ff, dim), (E, dim, ff)))
    corr = np.zeros(E, np.float32)
    corr[-1] = 50.0
    core = hc.MoeCore(router=_f32(np.zeros((E, dim)), cuda), correction=_torch(corr, cuda), gate=_f32(gate, cuda), up=_f32(up, cuda), down=_f32(down, cuda), shared=None, top=1,
                      groups=0, keep=0, scale=1.0, dtype=torch.bfloat16)
    y, rows, gather = core.forward(_torch(x, cuda, torch.bfloat16), form=2)
    got = _np(rows)[gather.cpu().numpy()[:, 0]] + _np(y)
    h = x.astype(np.float64)
    want = bf16_round((silu(h @ gate[-1].T) * (h @ up[-1].T)).astype(np.float32)).astype(np.float64) @ down[-1].T
    assert np.abs(got - want).max() <= TOL["bf16"] * np.abs(want).max()
    _status()
