"""The Zudisun section of the benchmark (`bench.py --only zudisun`): its mixers, its experts and a whole model at sizes that resemble a
real model's layers, random weights, beside the like kernels of the Nitenex and the Llama-style decoders at equal size.

Kernel figures as in hybrid_bench.py: median over timed calls, CUDA events on the launching stream, L2 flushed (256 MiB write) between
calls; `kernel_us` is the dominant kernel alone, `call_us` the whole core between its two projections.  Work counted: attention 2 FLOP
per multiply-add of q.k and of the values over visible pairs, plus the mixing of the heads (the wider product that replaces the mixing
and the low halves of split operands are not counted); scans and decode steps the bytes they must move once; experts the chosen ones'
products."""
from __future__ import annotations

import numpy as np

from . import capi
from .hybrid_bench import _generate, _timed, bench_like_decode, bench_like_prefill, bench_models as bench_like_models, bench_ssd

MODEL = dict(vocab=32000, width=2048, layers=24, ff=5632)
MAMBA = dict(inner=4096, state=16, dt_rank=128, conv=4)
ATTENTION = dict(heads=16, kv_heads=4, dim=128, vdim=128, scale=128 ** -0.5, bias_max=256, v_mix=True, q_temp=dict(coef=0.1, every=1024))
BIAS_ROWS = 32
MOE = dict(kind="moe", expert=dict(ff=704), router=dict(experts=64, top=6, scale=2.5, groups=dict(count=8, keep=4)), shared=dict(ff=1408))      # 5632 active hidden units


def model_config():
    m = MODEL
    layers = []
    for i in range(m["layers"]):                     # three state-space layers, then one of attention
        attn = i % 4 == 3
        layers.append(dict(type="attention" if attn else "mamba1", mixer=ATTENTION if attn else MAMBA, mlp=MOE if attn else dict(kind="dense", ff=m["ff"])))
    return dict(architecture="Zudisun", vocab=m["vocab"], width=m["width"], norm=dict(eps=1e-6), layers=layers)


def _randn(cx, g, *n):
    return cx.torch.randn(*n, generator=g, device=cx.dev)


def attention_core(cx, B, cap):
    from .hybrid_capi import SigmoidCore
    s = ATTENTION
    g = cx.torch.Generator(device=cx.dev).manual_seed(1)
    H = s["heads"]
    bias = _randn(cx, g, H, s["bias_max"]) - 4.0
    return SigmoidCore(H=H, G=s["kv_heads"], dim=s["dim"], vdim=s["vdim"], scale=s["scale"], eps=1e-6, talk=cx.torch.eye(H, device=cx.dev) + 0.1 * _randn(cx, g, H, H), bias=bias,
                       slots=B, cap=cap, dtype=cx.torch.bfloat16, temp_coef=s["q_temp"]["coef"], temp_every=s["q_temp"]["every"]), g


def bench_attention_prefill(cx, K, W, B, T):
    core, g = attention_core(cx, B, T)
    proj = core.proj_buffer(B * T)
    proj.normal_(generator=g)
    call_us, kern_us = _timed(cx, lambda: core.forward(proj, B, 0), K, W)
    s = core.s
    flops = 2.0 * B * s["H"] * T * (T + 1) / 2 * (s["dim"] + s["vdim"] + s["H"])
    tf = flops / kern_us / 1e6
    return dict(what=f"sigmoid prompt attention B={B} H={s['H']}/{s['G']} T={T}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us, tflops=tf, frac=tf / cx.peaks["tf"],
                bound="tensor")


def bench_attention_decode(cx, K, W, B, keys):
    torch = cx.torch
    core, g = attention_core(cx, B, keys)
    core.k_cache.normal_(generator=g)
    core.v_cache.normal_(generator=g)
    proj = core.proj_buffer(B)
    proj.normal_(generator=g)
    pos = torch.full((B,), keys - 1, dtype=torch.int32, device=cx.dev)
    call_us, kern_us = _timed(cx, lambda: core.forward(proj, B, 0, pos=pos, max_len=keys), K, W)
    s = core.s
    gbs = B * keys * s["G"] * (s["dim"] + s["vdim"]) * 2.0 / kern_us / 1e3
    return dict(what=f"sigmoid decode B={B} H={s['H']}/{s['G']} keys={keys}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us, gbs=gbs, frac=gbs / cx.peaks["hbm"], bound="hbm")


def bench_scan(cx, K, W, B, T):
    from .hybrid_capi import SelectiveCore
    torch, s = cx.torch, MAMBA
    g = torch.Generator(device=cx.dev).manual_seed(2)
    n, N, r, taps = s["inner"], s["state"], s["dt_rank"], s["conv"]
    R = lambda *d: _randn(cx, g, *d)
    core = SelectiveCore(inner=n, N=N, rank=r, taps=taps, conv_w=R(n, taps) * 0.5, conv_b=R(n) * 0.1, w_x=R(r + 2 * N, n) * n ** -0.5, w_dt=R(n, r) * r ** -0.5, dt_bias=R(n) - 3.0,
                         A=-torch.exp(R(n, N)), D=R(n), slots=B, dtype=torch.bfloat16)
    proj = torch.empty(B * T, 2 * n, dtype=torch.bfloat16, device=cx.dev).normal_(generator=g)
    pos = torch.full((B,), 7, dtype=torch.int32, device=cx.dev)
    call_us, kern_us = _timed(cx, lambda: core.forward(proj, B, pos), K, W)
    state = 2.0 * B * n * N * 4
    moved = state + (B * T * (2.0 * n + 4 * n + 2 * n + 2 * n + 4 * N) if T > 1 else B * 6.0 * n + 2.0 * n * r + 4.0 * n * N)      # x, dt, z, y, B and C; or x, z, y, W_dt, A
    gbs = moved / kern_us / 1e3
    return dict(what=f"selective scan B={B} T={T} inner={n} N={N}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us, gbs=gbs, frac=gbs / cx.peaks["hbm"], bound="hbm",
                gexp_per_s=B * T * n * N / kern_us / 1e3)


def bench_experts(cx, K, W, M, form=0):
    from .hybrid_capi import MoeCore, norm_add
    torch = cx.torch
    r, ff, sh, dim = MOE["router"], MOE["expert"]["ff"], MOE["shared"]["ff"], MODEL["width"]
    g = torch.Generator(device=cx.dev).manual_seed(3)
    R = lambda *d: _randn(cx, g, *d).mul_(d[-1] ** -0.5).to(torch.bfloat16)
    E = r["experts"]
    core = MoeCore(router=R(E, dim), correction=torch.zeros(E, device=cx.dev), gate=R(E, ff, dim), up=R(E, ff, dim), down=R(E, dim, ff), shared=(R(sh, dim), R(sh, dim), R(dim, sh)),
                   top=r["top"], groups=r["groups"]["count"], keep=r["groups"]["keep"], scale=r["scale"], dtype=torch.bfloat16)
    x = torch.empty(M, dim, dtype=torch.bfloat16, device=cx.dev).normal_(generator=g)
    h, w = torch.zeros(M, dim, device=cx.dev), torch.ones(dim, device=cx.dev)

    def call():
        y, rows, gather = core.forward(x, form=form)
        norm_add(h, y, w, 1e-6, rows=rows, gather=gather, copy=True)
    call_us, kern_us = _timed(cx, call, K, W)
    row = dict(what=f"experts M={M} E={E} top={r['top']} ff={ff} shared={sh}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us)
    active = 3 * dim * (r["top"] * ff + sh)
    if M > 256:
        tf = 2.0 * M * 3 * dim * r["top"] * ff / kern_us / 1e6                   # the bracketed kernels: the chosen experts' products
        row.update(tflops=tf, frac=tf / cx.peaks["tf"], call_tflops=2.0 * M * active / call_us / 1e6, bound="tensor")
    else:
        lg = x.float() @ core.router.float().T
        hit = torch.unique(torch.sigmoid(lg).topk(r["top"], dim=-1).indices).numel()
        grouped = core.last_kernel().startswith("linear")
        moved = 2.0 * 3 * dim * (hit * ff + (0 if grouped else sh))
        row.update(gbs=moved / kern_us / 1e3, frac=moved / kern_us / 1e3 / cx.peaks["hbm"], experts_hit=hit, bound="hbm")
    return row


def bench_projections(cx, K, W):
    """The layer's dense products; the kernels are those of the other decoders."""
    torch = cx.torch
    out, width, ff, n = [], MODEL["width"], MODEL["ff"], MAMBA["inner"]
    a = ATTENTION
    shapes = {"mamba in": (2 * n, width, capi.EPI_BF16), "mamba x": (MAMBA["dt_rank"] + 2 * MAMBA["state"], n, capi.EPI_BF16), "mamba dt": (n, MAMBA["dt_rank"], capi.EPI_F32),
              "mamba out": (width, n, capi.EPI_F32), "attention in": (a["heads"] * (a["dim"] + 1) + a["kv_heads"] * (a["dim"] + a["vdim"]), width, capi.EPI_BF16),
              "gate/up, ReLU gate": (2 * ff, width, capi.EPI_REGLU), "down": (width, ff, capi.EPI_F32),
              "gate/up, SwiGLU (Llama-style)": (2 * ff, width, capi.EPI_SWIGLU), "down (Llama-style)": (width, ff, capi.EPI_ADD_F32)}
    for M in (8, 4096):
        for name, (N, Kd, epi) in shapes.items():
            if name == "mamba dt" and M == 8:
                continue                                 # inside the scan kernel of a decode step
            x, w = torch.randn(M, Kd, device=cx.dev).to(torch.bfloat16), torch.randn(N, Kd, device=cx.dev).to(torch.bfloat16)
            cols = N // 2 if epi in (capi.EPI_SWIGLU, capi.EPI_REGLU) else N
            y = torch.zeros(M, (cols + 7) // 8 * 8, device=cx.dev, dtype=torch.float32 if epi in (capi.EPI_ADD_F32, capi.EPI_F32) else torch.bfloat16)
            us, _ = _timed(cx, lambda: capi.linear_ex(x, w, y, epilogue=epi), K, W)
            row = dict(what=f"{name} M={M} N={N} K={Kd}", call_us=us)
            if M <= 64:
                row.update(gbs=2.0 * N * Kd / us / 1e3, frac=2.0 * N * Kd / us / 1e3 / cx.peaks["hbm"], bound="hbm")
            else:
                row.update(tflops=2.0 * M * N * Kd / us / 1e6, frac=2.0 * M * N * Kd / us / 1e6 / cx.peaks["tf"], bound="tensor")
            out.append(row)
    return out


def bench_models(cx, reps=3, layers=None, like=True):
    from .model import model_from_config
    work = [(8, 512, 128), (1, 2048, 64), (32, 256, 64)]
    c = model_config()
    if layers:
        c["layers"] = c["layers"][:layers]
    m = model_from_config(c, "bfloat16", max_seq_len=4096)
    pool = np.random.default_rng(7).standard_normal(1 << 24, dtype=np.float32)
    n = active = 0
    for i, (name, s) in enumerate(m.param_shapes().items()):
        s = tuple(BIAS_ROWS if d < 0 else d for d in s)
        size = int(np.prod(s))
        w = 0.02 * np.resize(np.roll(pool, 977 * i) if size > pool.size else pool[(977 * i) % (pool.size - size + 1):][:size], s)
        if name.endswith(("norm", "norm1", "norm2", ".D")):
            w = w + 1.0
        elif name.endswith("dt.b"):
            w = w - 3.0
        elif name.endswith("mix.pb"):
            w = w - 5.0
        elif name.endswith("talk"):
            w = w + np.eye(s[0], dtype=np.float32)
        m.set_param(name, w)
        n += size
        active += size * (MOE["router"]["top"] / MOE["router"]["experts"] if ".mlp.e" in name else 1.0) if name != "embed" else 0
    out = dict(zudisun=dict(parameters=n, active_parameters=int(active), runs=[_generate(cx, m, c["vocab"], *x, reps) for x in work]), layers=len(c["layers"]))
    m.close()
    if like:
        out["like"] = bench_like_models(cx, reps, layers)
    return out


def bench_zudisun(cx, K=20, W=3, layers=None, part="all"):
    out = {}
    if part in ("all", "kernels"):
        out["kernels"] = [
            bench_like_prefill(cx, K, W, 4, 2048), bench_attention_prefill(cx, K, W, 4, 2048), bench_like_prefill(cx, K, W, 8, 512), bench_attention_prefill(cx, K, W, 8, 512),
            bench_like_prefill(cx, K, W, 1, 8192), bench_attention_prefill(cx, K, W, 1, 8192),
            bench_like_decode(cx, K, W, 128, 2304), bench_attention_decode(cx, K, W, 128, 2304), bench_like_decode(cx, K, W, 32, 2304), bench_attention_decode(cx, K, W, 32, 2304),
            bench_like_decode(cx, K, W, 8, 576), bench_attention_decode(cx, K, W, 8, 576),
            bench_ssd(cx, K, W, 8, 512), bench_scan(cx, K, W, 8, 512), bench_ssd(cx, K, W, 1, 4096), bench_scan(cx, K, W, 1, 4096), bench_ssd(cx, K, W, 4, 2048), bench_scan(cx, K, W, 4, 2048),
            bench_ssd(cx, K, W, 8, 1), bench_scan(cx, K, W, 8, 1), bench_ssd(cx, K, W, 64, 1), bench_scan(cx, K, W, 64, 1),
            bench_experts(cx, K, W, 4096), bench_experts(cx, K, W, 512), bench_experts(cx, K, W, 64), bench_experts(cx, K, W, 32, form=1), bench_experts(cx, K, W, 32, form=2),
            bench_experts(cx, K, W, 8, form=1), bench_experts(cx, K, W, 8, form=2), bench_experts(cx, K, W, 1)]
        out["projections"] = bench_projections(cx, K, W)
    if part in ("all", "models"):
        out["models"] = bench_models(cx, layers=layers)
    return out
