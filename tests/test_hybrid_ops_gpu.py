"""The operators of hybrid decoders (include/vesper_b200_hybrid.h) on the GPU against the plain equations of
hybrid_reference.py, one mechanism at a time.

Tolerances: fp32 forms 2e-5 of the largest output; bf16 forms 1.2e-2 (values are rounded to bf16 between steps on both
sides, at the same places, but an intermediate that lies on a rounding boundary may fall on either side)."""
import numpy as np
import pytest

import hybrid_reference as ref
from helpers import bf16_round

pytestmark = pytest.mark.gpu

TOL = {"f32": 2e-5, "bf16": 1.2e-2}


def _torch(x, cuda, dtype=None):
    import torch
    t = torch.from_numpy(np.ascontiguousarray(x)).to(cuda)
    return t.to(dtype) if dtype is not None else t


def _np(t):
    return t.detach().double().cpu().numpy()


def _dt(kind):
    import torch
    return torch.float32 if kind == "f32" else torch.bfloat16


def _close(got, want, tol):
    err = np.abs(_np(got) - want).max() / max(np.abs(want).max(), 1e-6)
    assert err <= tol, err


def _status():
    from vesper_b200 import capi
    capi.check_kernel_status(0)


# ---- embedding -----------------------------------------------------------------------------------

@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_embedding_with_bigram_rows_across_portions(cuda, kind):
    import torch
    from vesper_b200 import hybrid_capi as hc
    rng = np.random.default_rng(0)
    vocab, dim, buckets, mp, mc, B = 97, 40, 53, 31, 7, 3
    table, bigram = bf16_round(rng.standard_normal((vocab, dim))), bf16_round(rng.standard_normal((buckets + 1, dim)))
    add, scale = rng.standard_normal(dim).astype(np.float32), rng.standard_normal(dim).astype(np.float32)
    ids = rng.integers(0, vocab, (B, 14))
    slots = np.array([4, 0, 2], np.int32)
    lens = torch.zeros(B, dtype=torch.int32, device=cuda)
    prev = torch.full((5,), 1 << 20, dtype=torch.int32, device=cuda)         # whatever a slot held before: unused at position 0
    at = 0
    for T in (1, 2, 6, 1, 4):
        h, e, xs, step = hc.embed_sequence(_torch(ids[:, at:at + T].astype(np.int32), cuda), _torch(table, cuda, _dt(kind)), lens, prev,
                                           bigram=_torch(bigram, cuda, _dt(kind)), buckets=buckets, mul_prev=mp, mul_cur=mc, slots=_torch(slots, cuda),
                                           add=_torch(add, cuda), scale=_torch(scale, cuda), want_copy=True)
        want = np.concatenate([table[ids[b, at:at + T]] + bigram[ref.bigram_rows(ids[b, at:at + T], ids[b, at - 1] if at else None, buckets, mp, mc)] for b in range(B)])
        assert step.cpu().tolist() == [at] * B
        assert np.abs(_np(e) - want).max() <= 1e-6 and np.abs(_np(h) - (want + add)).max() <= 1e-6
        assert np.abs(_np(xs) - (want + add) * scale).max() <= 2 ** -8 * np.abs((want + add) * scale).max()
        at += T
        assert lens.cpu().tolist() == [at] * B and prev.cpu()[slots.tolist()].tolist() == ids[:, at - 1].tolist()
    _status()


def test_residual_add_and_rms_norm(cuda):
    import torch
    from vesper_b200 import capi, hybrid_capi as hc
    rng = np.random.default_rng(1)
    M, dim, count = 7, 48, 45
    h, e = rng.standard_normal((M, dim)).astype(np.float32), rng.standard_normal((M, dim)).astype(np.float32)
    v, g = rng.standard_normal(dim).astype(np.float32), rng.standard_normal(dim).astype(np.float32)
    ht, et, vt, gt = (_torch(x, cuda) for x in (h, e, v, g))
    xs = torch.empty(M, dim, dtype=torch.bfloat16, device=cuda)
    capi.check(hc.load().vb200_residual_add(0, hc._stream(), ht.data_ptr(), et.data_ptr(), vt.data_ptr(), M, dim, gt.data_ptr(), xs.data_ptr()))
    want = h.astype(np.float64) + e + v
    assert np.abs(_np(ht) - want).max() <= 1e-6 and np.abs(_np(xs) - want * g).max() <= 2 ** -8 * np.abs(want * g).max()
    h[:, count:] = 0                                     # padding columns
    ht, out = _torch(h, cuda), torch.empty(M, dim, device=cuda)
    capi.check(hc.load().vb200_rms_norm_f32(0, hc._stream(), ht.data_ptr(), gt.data_ptr(), out.data_ptr(), M, dim, count, 1e-3))
    want = ref.rms_norm(h[:, :count].astype(np.float64), 1e-3) * g[:count]
    assert np.abs(_np(out)[:, :count] - want).max() <= 1e-5


@pytest.mark.parametrize("M", [1, 5, 40, 64, 65, 300])
@pytest.mark.parametrize("N,K", [(96, 64), (200, 136)])
def test_linear_squared_relu_and_second_addend(cuda, M, N, K):
    import torch
    from vesper_b200 import capi, hybrid_capi as hc
    rng = np.random.default_rng(2)
    x, w = bf16_round(rng.standard_normal((M, K))), bf16_round(rng.standard_normal((N, K)) / np.sqrt(K))
    bias, add, h = (rng.standard_normal(s).astype(np.float32) for s in (N, (M, N), (M, N)))
    acc = x.astype(np.float64) @ w.T.astype(np.float64)
    xt, wt = _torch(x, cuda, torch.bfloat16), _torch(w, cuda, torch.bfloat16)
    out = torch.zeros(M, N, dtype=torch.bfloat16, device=cuda)
    capi.linear_ex(xt, wt, out, epilogue=capi.EPI_RELU2)
    _close(out, ref.squared_relu(acc), 5e-3)
    ht, at, bt = _torch(h, cuda), _torch(add, cuda), _torch(bias, cuda)
    capi.linear_ex(xt, wt, ht, epilogue=capi.EPI_ADD_F32, bias=bt, addend=at)
    _close(ht, h + acc + bias + add, 1e-5)
    xf, wf, hf, of = _torch(x, cuda), _torch(w, cuda), _torch(h, cuda), torch.zeros(M, N, device=cuda)
    L, s = hc.load(), hc._stream()
    capi.check(L.vb200_linear_f32_ex(0, s, xf.data_ptr(), K, wf.data_ptr(), K, bt.data_ptr(), at.data_ptr(), hf.data_ptr(), N, M, N, K, capi.EPI_ADD_F32))
    _close(hf, h + acc + bias + add, 1e-6)
    capi.check(L.vb200_linear_f32_ex(0, s, xf.data_ptr(), K, wf.data_ptr(), K, None, None, of.data_ptr(), N, M, N, K, capi.EPI_RELU2))
    _close(of, ref.squared_relu(acc), 1e-6)
    _status()


# ---- latent attention ----------------------------------------------------------------------------

# sizes: one head, parts that differ from a multiple of 16 / 64, more heads than one 16-row tile, windows below, at and
# above a 64-key block and a 32-key tile, rank of several boxes
LATENT = {
    "small": dict(H=3, dim=24, rot_dim=8, vdim=40, rank=56, window=37),
    "one": dict(H=1, dim=8, rot_dim=2, vdim=8, rank=20, window=5),
    "odd": dict(H=2, dim=20, rot_dim=6, vdim=12, rank=33, window=64),
    "wide": dict(H=18, dim=128, rot_dim=64, vdim=128, rank=512, window=150),
    "mid": dict(H=5, dim=72, rot_dim=24, vdim=80, rank=136, window=65),
    "rank256": dict(H=4, dim=64, rot_dim=32, vdim=64, rank=256, window=128),
    "self": dict(H=4, dim=16, rot_dim=16, vdim=16, rank=32, window=1),
}


class LatentCase:
    def __init__(self, cuda, kind, sizes, slots=1, seed=0, sink=True, max_len=None, gain=1.0):
        from vesper_b200.hybrid_capi import LatentCore
        self.cuda, self.kind, self.s = cuda, kind, sizes
        rng = self.rng = np.random.default_rng(seed)
        H, dim, rot, vdim, rank = (sizes[k] for k in ("H", "dim", "rot_dim", "vdim", "rank"))
        self.rnd = bf16_round if kind == "bf16" else (lambda x: np.asarray(x, np.float32))
        self.base, self.eps = 900.0, 1e-5
        self.scale = gain / np.sqrt(dim + rot)
        self.expand = bf16_round(rng.standard_normal((H * (dim + vdim), rank)) / np.sqrt(rank))
        self.c_norm = (1 + 0.2 * rng.standard_normal(rank)).astype(np.float32)
        self.sink = (1.5 * rng.standard_normal(H)).astype(np.float32) if sink else None
        f = self.base ** (-2.0 * np.arange(rot // 2) / rot)
        self.core = LatentCore(inv_freq=f, scale=float(self.scale), eps=self.eps, expand=_torch(self.expand, cuda, _dt(kind)), c_norm=_torch(self.c_norm, cuda),
                               sink=None if self.sink is None else _torch(self.sink, cuda), slots=slots, max_len=max_len, **sizes)

    def sequence(self, L):
        """Projections of a sequence [L, cols], as the input GEMM would leave them."""
        return self.rnd(self.rng.standard_normal((L, self.core.proj_cols)))

    def want(self, seq):
        """Whole sequence by the equations, bf16 rounding where the product path stores bf16."""
        s, r = self.s, lambda x: self.rnd(x.astype(np.float32)).astype(np.float64)
        H, dim, rot, vdim, rank = (s[k] for k in ("H", "dim", "rot_dim", "vdim", "rank"))
        L, x, pos = len(seq), seq.astype(np.float64), np.arange(len(seq))
        q = x[:, :H * (dim + rot)].reshape(L, H, dim + rot)
        q = np.concatenate([q[..., :dim], r(ref.rotate_half(q[..., dim:], pos, self.base))], -1)
        c = r(ref.rms_norm(x[:, H * (dim + rot):-rot], self.eps) * self.c_norm)
        kr = r(ref.rotate_half(x[:, None, -rot:], pos, self.base))
        kv = r(c @ self.expand.T.astype(np.float64))
        k = np.concatenate([kv[:, :H * dim].reshape(L, H, dim), np.repeat(kr, H, 1)], -1)
        return ref.window_attention_with_sink(q, k, kv[:, H * dim:].reshape(L, H, vdim), pos, pos, self.scale, s["window"], self.sink).reshape(L, H * vdim)

    def run(self, seq, cuts, slot=None):
        """The sequence in portions; one token goes through decode.  Returns [L, H*vdim]."""
        import torch
        outs, at = [], 0
        slots = None if slot is None else torch.tensor([slot], dtype=torch.int32, device=self.cuda)
        for T in cuts:
            proj = self.core.proj_buffer(T)
            proj[:, :self.core.proj_cols] = _torch(seq[at:at + T], self.cuda, _dt(self.kind))
            if T > 1:
                outs.append(self.core.prefill(proj, 1, at, slots=slots))
            else:
                outs.append(self.core.decode(proj, torch.tensor([at], dtype=torch.int32, device=self.cuda), slots=slots))
            at += T
        _status()
        return torch.cat(outs)


def _cuts(L, plan):
    out = []
    while sum(out) < L:
        out.append(min(plan[len(out) % len(plan)], L - sum(out)))
    return out


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(LATENT))
def test_latent_attention_whole_portions_and_tokens(cuda, kind, name):
    c = LatentCase(cuda, kind, LATENT[name], seed=len(name))
    L = min(2 * LATENT[name]["window"] + 40, 260)
    seq = c.sequence(L)
    want = c.want(seq)
    _close(c.run(seq, [L]), want, TOL[kind])
    tuned = kind == "bf16" and name not in ("odd", "one")
    assert c.core.last_kernel() == ("latent_prefill_sm100_kernel" if tuned else "latent_prefill_generic_kernel")
    _close(c.run(seq, _cuts(L, [2, 19, 3, 64, 1, 2, 1, 1, 50])), want, TOL[kind])
    _close(c.run(seq, [L - 20] + [1] * 20), want, TOL[kind])
    assert c.core.last_kernel() == ("latent_split_mma_kernel" if kind == "bf16" else "latent_split_generic_kernel")


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("window", [2, 31, 32, 33, 63, 64, 65, 130])
def test_window_edges_show(cuda, kind, window):
    """A key just inside the window takes nearly all the weight of its query; one step further out it is not seen.
    The loud key meets every query at both distances, in prompts, portions and decoded tokens."""
    s = dict(H=2, dim=16, rot_dim=8, vdim=16, rank=16, window=window)
    c = LatentCase(cuda, kind, s, seed=window, gain=1.0)
    L = 2 * window + 70
    seq = c.sequence(L)
    H, dim, rot = 2, 16, 8
    loud = [5, window + 9]
    for j in loud:                                   # query at distance window - 1 (inside) and window (outside)
        cl = ref.rms_norm(seq[j, H * (dim + rot):-rot].astype(np.float64), c.eps) * c.c_norm
        for i in (j + window - 1, j + window):
            for h in range(H):
                k = c.expand[h * dim:(h + 1) * dim].astype(np.float64) @ cl
                seq[i, h * (dim + rot):h * (dim + rot) + dim] = c.rnd(60.0 * k / (k @ k))
    want = c.want(seq)
    for j in loud:                                   # the planted pair does decide the output
        assert np.abs(want[j + window - 1] - want[j + window]).max() > 0.05
    for cuts in ([L], _cuts(L, [7, 2, window, 1]), [3] + [1] * (L - 3)):
        _close(c.run(seq, cuts), want, TOL[kind])


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_sink_is_counted_once_and_optional(cuda, kind):
    for sink in (True, False):
        c = LatentCase(cuda, kind, LATENT["small"], seed=3, sink=sink)
        if sink:
            c.sink[:] = [-20.0, 0.0, 9.0]            # none, some and nearly all of the weight
            c.core.sink.copy_(_torch(c.sink, cuda))
        seq = c.sequence(90)
        want = c.want(seq)
        for cuts in ([90], [70] + [1] * 20, [1] * 12):
            n = sum(cuts)
            _close(c.run(seq[:n], cuts), want[:n], TOL[kind])


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_latent_slots_are_reused_and_batches_do_not_mix(cuda, kind):
    import torch
    c = LatentCase(cuda, kind, LATENT["rank256"], slots=4, seed=8)
    seqs = [c.sequence(n) for n in (150, 90, 40)]
    wants = [c.want(s) for s in seqs]
    _close(c.run(seqs[0], [150], slot=2), wants[0], TOL[kind])
    c.core.cache[2] *= 64.0                          # what a finished sequence left behind is never read
    _close(c.run(seqs[1], _cuts(90, [1, 1, 2, 30, 1]), slot=2), wants[1], TOL[kind])
    # a decode batch of unequal lengths in scattered slots, against each alone
    slots = torch.tensor([3, 0, 1], dtype=torch.int32, device=cuda)
    for i, s in enumerate(seqs):
        c.run(s[:-4], [len(s) - 4], slot=int(slots[i]))
    for t in range(4):
        proj = c.core.proj_buffer(3)
        for i, s in enumerate(seqs):
            proj[i, :c.core.proj_cols] = _torch(s[len(s) - 4 + t], cuda, _dt(kind))
        pos = torch.tensor([len(s) - 4 + t for s in seqs], dtype=torch.int32, device=cuda)
        out = c.core.decode(proj, pos, slots=slots)
        for i, s in enumerate(seqs):
            _close(out[i], wants[i][len(s) - 4 + t], TOL[kind])
    # a prompt batch
    proj = c.core.proj_buffer(2 * 40)
    for i in range(2):
        proj[40 * i:40 * i + 40, :c.core.proj_cols] = _torch(seqs[i][:40], cuda, _dt(kind))
    out = c.core.prefill(proj, 2, 0, slots=slots[:2].contiguous())
    for i in range(2):
        _close(out[40 * i:40 * i + 40], wants[i][:40], TOL[kind])
    _status()


def test_ring_shorter_than_the_window(cuda):
    """Sequences known to be short get a ring of their longest length; the window then never cuts."""
    c = LatentCase(cuda, "bf16", dict(LATENT["small"], window=1000), seed=5, max_len=120)
    seq = c.sequence(120)
    _close(c.run(seq, [60, 2] + [1] * 58), c.want(seq), TOL["bf16"])


def test_far_positions_rotate_exactly(cuda):
    """Angles at positions where fp32 position * frequency would be off by several hundredths of a turn."""
    import torch
    c = LatentCase(cuda, "f32", LATENT["small"], seed=6)
    start, T = 3_000_000, 12
    seq = c.sequence(T)
    proj = c.core.proj_buffer(T)
    proj[:, :c.core.proj_cols] = _torch(seq, cuda)
    c.core.prefill(proj, 1, start, pos=torch.tensor([start], dtype=torch.int32, device=cuda))
    H, dim, rot = 3, 24, 8
    q = seq[:, :H * (dim + rot)].reshape(T, H, dim + rot).astype(np.float64)
    want = ref.rotate_half(q[..., dim:], np.arange(start, start + T), c.base)
    assert np.abs(_np(proj[:, :H * (dim + rot)].reshape(T, H, dim + rot)[..., dim:]) - want).max() <= 2e-5


# ---- Mamba-2 -------------------------------------------------------------------------------------

SSD = {
    "small": dict(H=6, P=24, N=16, G=2, taps=4, norm_groups=3),
    "one": dict(H=1, P=8, N=8, G=1, taps=1, norm_groups=1),
    "odd": dict(H=3, P=10, N=12, G=3, taps=3, norm_groups=1),
    "real": dict(H=4, P=64, N=128, G=1, taps=4, norm_groups=2),
    "wide": dict(H=2, P=136, N=72, G=2, taps=2, norm_groups=2),
    "deep": dict(H=2, P=40, N=200, G=1, taps=5, norm_groups=1),
}


class SsdCase:
    def __init__(self, cuda, kind, sizes, slots=1, seed=0):
        from vesper_b200.hybrid_capi import SsdCore
        self.cuda, self.kind, self.s, self.eps = cuda, kind, sizes, 1e-5
        rng = self.rng = np.random.default_rng(seed)
        H, P, N, G, taps = (sizes[k] for k in ("H", "P", "N", "G", "taps"))
        ch = H * P + 2 * G * N
        f = lambda x: np.asarray(x, np.float32)
        self.w = dict(conv_w=f(rng.standard_normal((ch, taps)) / np.sqrt(taps)), conv_b=f(0.1 * rng.standard_normal(ch)), dt_bias=f(rng.standard_normal(H) - 2.0),
                      A_log=f(np.log(rng.uniform(0.3, 4.0, H))), D=f(rng.standard_normal(H)), norm_w=f(1 + 0.2 * rng.standard_normal(H * P)))
        self.rnd = bf16_round if kind == "bf16" else f
        self.core = SsdCore(eps=self.eps, slots=slots, dtype=_dt(kind), **sizes, **{k: _torch(v, cuda) for k, v in self.w.items()})

    def sequence(self, L):
        return self.rnd(self.rng.standard_normal((L, self.core.proj_cols)))

    def want(self, seq):
        H, P, N, G, taps, ng = (self.s[k] for k in ("H", "P", "N", "G", "taps", "norm_groups"))
        w = {k: v.astype(np.float64) for k, v in self.w.items()}
        x, inner, T = seq.astype(np.float64), H * P, len(seq)
        conv, _ = ref.causal_conv(x[:, inner:2 * inner + 2 * G * N], np.zeros((taps - 1, inner + 2 * G * N)), w["conv_w"], w["conv_b"])
        xbc = self.rnd(ref.silu(conv).astype(np.float32)).astype(np.float64)
        dt = ref.softplus(x[:, 2 * inner + 2 * G * N:] + w["dt_bias"])
        y, _ = ref.ssd_scan(xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N), dt,
                            w["A_log"], w["D"], np.zeros((H, N, P)))
        return ref.gated_group_norm(y.reshape(T, inner), x[:, :inner], w["norm_w"], ng, self.eps)

    def run(self, seq, cuts, slot=None, form=0):
        import torch
        outs, at = [], 0
        slots = None if slot is None else torch.tensor([slot], dtype=torch.int32, device=self.cuda)
        for T in cuts:
            proj = self.core.proj_buffer(T)
            proj[:, :self.core.proj_cols] = _torch(seq[at:at + T], self.cuda, _dt(self.kind))
            outs.append(self.core.forward(proj, 1, torch.tensor([at], dtype=torch.int32, device=self.cuda), slots=slots, form=form))
            at += T
        _status()
        return torch.cat(outs)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
@pytest.mark.parametrize("name", sorted(SSD))
def test_ssd_whole_portions_and_tokens(cuda, kind, name):
    c = SsdCase(cuda, kind, SSD[name], seed=len(name))
    L = 230
    seq = c.sequence(L)
    want = c.want(seq)
    _close(c.run(seq, [L]), want, TOL[kind])
    chunked = kind == "bf16" and name != "odd"
    walk = chunked and SSD[name]["P"] <= 64 and SSD[name]["N"] <= 128
    assert c.core.last_kernel() == ("ssd_walk_sm100_kernel" if walk else "ssd_chunk_kernel" if chunked else "ssd_scan_kernel")
    _close(c.run(seq, _cuts(L, [2, 64, 3, 1, 1, 63, 2, 65, 17])), want, TOL[kind])
    _close(c.run(seq, [L - 40] + [1] * 40), want, TOL[kind])
    _close(c.run(seq[:30], [1] * 30), want[:30], TOL[kind])
    if chunked:                                      # token by token and chunked forms agree, whatever the portion
        _close(c.run(seq, [L], form=1), want, TOL[kind])
        _close(c.run(seq, _cuts(L, [2, 5, 9, 70]), form=2), want, TOL[kind])
        _close(c.run(seq, _cuts(L, [129, 98]), form=2), want, TOL[kind])
        _close(c.run(seq, _cuts(L, [3, 200]), form=3), want, TOL[kind])
        assert c.core.last_kernel() == "ssd_chunk_kernel"


def test_ssd_state_is_fp32_class_over_a_long_prompt(cuda):
    """Slow decays: the state sums hundreds of tokens.  The bf16 form's state must match an fp64 recurrence on the same
    (bf16) inputs far below bf16 rounding: the decays, weights and state never pass through a single bf16 value."""
    import torch
    c = SsdCase(cuda, "bf16", dict(H=2, P=64, N=64, G=1, taps=1, norm_groups=1), seed=4)
    c.w["A_log"][:] = np.log([1e-3, 5e-2])
    c.core.w["A_log"].copy_(_torch(c.w["A_log"], cuda))
    c.core.w["conv_w"].fill_(1.0)
    c.core.w["conv_b"].zero_()
    seq = c.sequence(900)
    outs = None
    for form, cuts in ((2, [900]), (2, [333, 567]), (3, [900]), (1, [900])):
        out = c.run(seq, cuts, form=form)
        outs = out if form == 2 and len(cuts) == 1 else outs
        _close(out, _np(outs), TOL["bf16"])                  # segments, portions and tokens give the same outputs
        x = ref.silu(seq.astype(np.float64)[:, 128:384])
        x = bf16_round(x.astype(np.float32)).astype(np.float64)
        dt = ref.softplus(seq.astype(np.float64)[:, 384:] + c.w["dt_bias"])
        _, S = ref.ssd_scan(x[:, :128].reshape(-1, 2, 64), x[:, 128:192].reshape(-1, 1, 64), x[:, 192:].reshape(-1, 1, 64), dt,
                            c.w["A_log"].astype(np.float64), c.w["D"].astype(np.float64), np.zeros((2, 64, 64)))
        got = _np(c.core.state[0])
        flips = np.abs(got - S).max() / np.abs(S).max()      # a convolution output on a rounding boundary may differ by one bf16 step
        rms = np.sqrt(((got - S) ** 2).mean()) / np.sqrt((S ** 2).mean())
        assert rms <= 2e-4 and flips <= 2e-3, (form, rms, flips)


@pytest.mark.parametrize("kind", ["f32", "bf16"])
def test_ssd_slots_are_reused_and_batches_do_not_mix(cuda, kind):
    import torch
    c = SsdCase(cuda, kind, SSD["small"], slots=4, seed=9)
    seqs = [c.sequence(n) for n in (100, 61, 33)]
    wants = [c.want(s) for s in seqs]
    c.core.state.fill_(1e30)
    c.core.conv_state.fill_(1e3)
    _close(c.run(seqs[0], [100], slot=3), wants[0], TOL[kind])
    _close(c.run(seqs[1], _cuts(61, [1, 1, 2, 30]), slot=3), wants[1], TOL[kind])
    slots = torch.tensor([2, 3, 0], dtype=torch.int32, device=cuda)
    for i, s in enumerate(seqs):
        c.run(s[:-5], [len(s) - 5], slot=int(slots[i]))
    for t in range(5):
        proj = c.core.proj_buffer(3)
        for i, s in enumerate(seqs):
            proj[i, :c.core.proj_cols] = _torch(s[len(s) - 5 + t], cuda, _dt(kind))
        out = c.core.forward(proj, 3, torch.tensor([len(s) - 5 + t for s in seqs], dtype=torch.int32, device=cuda), slots=slots)
        for i, s in enumerate(seqs):
            _close(out[i], wants[i][len(s) - 5 + t], TOL[kind])
    for T in (2, 33):                                # prompt batches, both forms
        proj = c.core.proj_buffer(3 * T)
        for i in range(3):
            proj[T * i:T * i + T, :c.core.proj_cols] = _torch(seqs[i][:T], cuda, _dt(kind))
        out = c.core.forward(proj, 3, torch.zeros(3, dtype=torch.int32, device=cuda), slots=slots)
        for i in range(3):
            _close(out[T * i:T * i + T], wants[i][:T], TOL[kind])
    _status()
