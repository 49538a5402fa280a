"""The hybrid section of the benchmark (`bench.py --only hybrid`): the hybrid decoder's mixers and whole model at sizes
that resemble a real model's layers, random weights, beside the Llama-style decoder at equal size.

Kernel figures: median over timed calls, CUDA events on the launching stream, L2 flushed (256 MiB write) between calls;
`kernel_us` is the dominant kernel alone (event brackets inside the library, a pass of its own), `call_us` the whole
mixer core between its two projections.  Work counted: 2 FLOP per multiply-add of the attention products over visible
(query, key) pairs (the low halves of split operands are not counted); bytes = what the operator must move once."""
from __future__ import annotations

import numpy as np

from . import capi

# width, layers and feed-forward as in the Llama-style workload; a squared-ReLU feed-forward of 3/2 the width has SwiGLU's parameters
MODEL = dict(vocab=32000, width=2048, layers=24, ff=8448, window=1024)
MAMBA = dict(heads=64, vdim=64, state=128, groups=1, conv=4, norm_groups=1)
LATENT = dict(heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512, scale=192 ** -0.5, rot=dict(base=10000.0, dims=64))


def model_config():
    m = MODEL
    layers = []
    for i in range(m["layers"]):                     # three state-space layers, then one of attention
        attn = i % 4 == 3
        layers.append(dict(type="latent_attention" if attn else "mamba2", mixer=dict(LATENT, mask=dict(size=m["window"])) if attn else MAMBA,
                           mlp=dict(kind="dense", ff=m["ff"])))
    return dict(architecture="Nitenex", vocab=m["vocab"], width=m["width"], norm=dict(eps=1e-6), layers=layers,
                embedding=dict(bigram=dict(buckets=65536, mul_prev=31337, mul_cur=1)))


def _timed(cx, call, K, W, before=None):
    """(median microseconds of a call, of its dominant kernel)."""
    torch = cx.torch
    for _ in range(W):
        if before:
            before()
        call()
    cx.sync_all()
    t = []
    for _ in range(K):
        if before:
            before()
        cx.flush_l2()
        a, b = cx.event(), cx.event()
        a.record(); call(); b.record()
        torch.cuda.synchronize()
        t.append(a.elapsed_time(b) * 1e3)
    capi.profile_enable(True)
    k = []
    for _ in range(min(K, 10)):
        if before:
            before()
        cx.flush_l2()
        call()
        torch.cuda.synchronize()
        ms, n = capi.profile_read()
        k.append(ms * 1e3 - sum(k))                  # the reading is a running total
    capi.profile_enable(False)
    capi.check_kernel_status(cx.local)
    return float(np.median(t)), float(np.median(k))


def latent_core(cx, B, window, H=None):
    from .hybrid_capi import LatentCore
    torch, s = cx.torch, LATENT
    H = H or s["heads"]
    g = torch.Generator(device=cx.dev).manual_seed(1)
    f = s["rot"]["base"] ** (-2.0 * np.arange(s["rot_dim"] // 2) / s["rot_dim"])
    expand = torch.randn(H * (s["dim"] + s["vdim"]), s["kv_rank"], generator=g, device=cx.dev).mul_(s["kv_rank"] ** -0.5).to(torch.bfloat16)
    return LatentCore(H=H, dim=s["dim"], rot_dim=s["rot_dim"], vdim=s["vdim"], rank=s["kv_rank"], window=window, scale=s["scale"], eps=1e-6, inv_freq=f, expand=expand,
                      c_norm=torch.ones(s["kv_rank"], device=cx.dev), sink=torch.zeros(H, device=cx.dev), slots=B), g


def ssd_core(cx, B):
    from .hybrid_capi import SsdCore
    torch, s = cx.torch, MAMBA
    g = torch.Generator(device=cx.dev).manual_seed(2)
    ch, H = s["heads"] * s["vdim"] + 2 * s["groups"] * s["state"], s["heads"]
    r = lambda *n: torch.randn(*n, generator=g, device=cx.dev)
    return SsdCore(H=H, P=s["vdim"], N=s["state"], G=s["groups"], taps=s["conv"], norm_groups=s["norm_groups"], eps=1e-6, conv_w=r(ch, s["conv"]) * 0.5, conv_b=r(ch) * 0.1,
                   dt_bias=r(H) - 3.0, A_log=r(H) * 0.5, D=r(H), norm_w=torch.ones(H * s["vdim"], device=cx.dev), slots=B, dtype=torch.bfloat16), g


def bench_latent_prefill(cx, K, W, B, T, window, H=None):
    torch = cx.torch
    core, g = latent_core(cx, B, window, H)
    H = core.s["H"]
    proj = core.proj_buffer(B * T)
    proj.normal_(generator=g)
    call_us, kern_us = _timed(cx, lambda: core.prefill(proj, B, 0), K, W)
    pairs = sum(min(i + 1, window) for i in range(T))
    flops = 2.0 * B * H * pairs * (core.s["dim"] + core.s["rot_dim"] + core.s["vdim"])
    tf = flops / kern_us / 1e6
    return dict(what=f"latent prompt attention B={B} H={H} T={T} window={window}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us, tflops=tf,
                frac=tf / cx.peaks["tf"], bound="tensor")


def bench_latent_decode(cx, K, W, B, keys, H=None):
    torch = cx.torch
    core, g = latent_core(cx, B, keys, H)
    core.cache.normal_(generator=g)
    proj = core.proj_buffer(B)
    proj.normal_(generator=g)
    pos = torch.full((B,), keys + 5, dtype=torch.int32, device=cx.dev)
    call_us, kern_us = _timed(cx, lambda: core.decode(proj, pos), K, W)
    gbs = B * keys * core.ldc * 2.0 / kern_us / 1e3
    return dict(what=f"latent decode B={B} H={core.s['H']} keys={keys}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us, gbs=gbs, frac=gbs / cx.peaks["hbm"], bound="hbm")


def bench_ssd(cx, K, W, B, T):
    torch = cx.torch
    core, g = ssd_core(cx, B)
    proj = core.proj_buffer(B * T)
    proj.normal_(generator=g)
    pos = torch.full((B,), 7, dtype=torch.int32, device=cx.dev)
    call_us, kern_us = _timed(cx, lambda: core.forward(proj, B, pos), K, W)
    s = core.s
    inner, gn = s["H"] * s["P"], s["G"] * s["N"]
    state = 2.0 * B * s["H"] * s["N"] * s["P"] * 4                          # read and written
    if T == 1:
        moved = state + B * 2.0 * (2 * inner + 2 * gn + s["H"]) + B * 4.0 * inner
    else:
        moved = state + B * T * 2.0 * (inner + 2 * gn + inner + inner + s["H"])   # x, B, C; z; y; dt
    gbs = moved / kern_us / 1e3
    # what the recurrence costs as products: C S, B^T x, and the causal halves of C B^T and (.) x, per 64-token chunk
    flops = 2.0 * B * T * s["H"] * (2 * s["N"] * s["P"] + 33 * (s["N"] + s["P"])) if T > 1 else 4.0 * B * s["H"] * s["N"] * s["P"]
    return dict(what=f"state-space mixer B={B} T={T} H={s['H']} P={s['P']} N={s['N']}", kernel=core.last_kernel(), kernel_us=kern_us, call_us=call_us, gbs=gbs,
                frac=gbs / cx.peaks["hbm"], tflops=flops / kern_us / 1e6, bound="hbm")


def bench_like_prefill(cx, K, W, B, T):
    """The Llama-style decoder's prompt attention (16 query / 4 KV heads of 128, RoPE and append fused) at the same batch and length."""
    torch = cx.torch
    g = torch.Generator(device=cx.dev).manual_seed(4)
    r = lambda *n: torch.randn(*n, generator=g, device=cx.dev, dtype=torch.bfloat16)
    q, k, v = r(B, 16, T, 128), r(B, 4, T, 128), r(B, 4, T, 128)
    o, kc, vc = torch.empty_like(q), torch.zeros_like(k), torch.zeros_like(v)
    call_us, kern_us = _timed(cx, lambda: capi.prefill(q, k, v, o, None, scale=128 ** -0.5, causal=True, theta=10000.0, k_cache=kc, v_cache=vc), K, W)
    tf = 4.0 * B * 16 * 128 * T * (T + 1) / 2 / kern_us / 1e6
    return dict(what=f"like kernel: GQA prompt attention B={B} H=16/4 T={T} D=128", kernel="prefill_sm100_kernel", kernel_us=kern_us, call_us=call_us, tflops=tf,
                frac=tf / cx.peaks["tf"], bound="tensor")


def bench_like_decode(cx, K, W, B, keys):
    """The Llama-style decoder's decode attention (16 query / 4 KV heads of 128)."""
    torch = cx.torch
    g = torch.Generator(device=cx.dev).manual_seed(5)
    r = lambda *n: torch.randn(*n, generator=g, device=cx.dev, dtype=torch.bfloat16)
    q, k1, v1 = r(B, 16, 1, 128), r(B, 4, 1, 128), r(B, 4, 1, 128)
    kc, vc, o = r(B, 4, keys, 128), r(B, 4, keys, 128), torch.empty_like(q)
    seq = torch.full((B,), keys - 1, dtype=torch.int32, device=cx.dev)
    call_us, kern_us = _timed(cx, lambda: capi.decode(q, o, kc, vc, scale=128 ** -0.5, k_new=k1, v_new=v1, theta=10000.0, seq_lens=seq, max_len=keys), K, W)
    gbs = B * keys * 4 * 128 * 2 * 2.0 / kern_us / 1e3
    return dict(what=f"like kernel: GQA decode B={B} H=16/4 keys={keys} D=128", kernel="decode_gqa_mma_kernel", kernel_us=kern_us, call_us=call_us, gbs=gbs,
                frac=gbs / cx.peaks["hbm"], bound="hbm")


def bench_projections(cx, K, W):
    """The layer's GEMMs at decode and prompt sizes, which both decoders share."""
    torch = cx.torch
    out = []
    width, ff = MODEL["width"], MODEL["ff"]
    inner = MAMBA["heads"] * MAMBA["vdim"]
    shapes = {"mamba in": (2 * inner + 2 * MAMBA["groups"] * MAMBA["state"] + MAMBA["heads"], width, capi.EPI_BF16), "mamba out": (width, inner, capi.EPI_ADD_F32),
              "latent in": (LATENT["heads"] * 192 + 576, width, capi.EPI_BF16), "latent out": (width, 2048, capi.EPI_ADD_F32), "up, squared ReLU": (ff, width, capi.EPI_RELU2),
              "down": (width, ff, capi.EPI_ADD_F32), "gate/up, SwiGLU (Llama-style)": (2 * 5632, width, capi.EPI_SWIGLU), "down (Llama-style)": (width, 5632, capi.EPI_ADD_F32)}
    for M in (8, 4096):
        for name, (N, Kd, epi) in shapes.items():
            x = torch.randn(M, Kd, device=cx.dev).to(torch.bfloat16)
            w = torch.randn(N, Kd, device=cx.dev).to(torch.bfloat16)
            cols = N // 2 if epi == capi.EPI_SWIGLU else N
            y = torch.zeros(M, (cols + 7) // 8 * 8, device=cx.dev, dtype=torch.float32 if epi == capi.EPI_ADD_F32 else torch.bfloat16)
            us, _ = _timed(cx, lambda: capi.linear_ex(x, w, y, epilogue=epi), K, W)
            row = dict(what=f"{name} M={M} N={N} K={Kd}", call_us=us)
            if M <= 64:
                row.update(gbs=2.0 * N * Kd / us / 1e3, frac=2.0 * N * Kd / us / 1e3 / cx.peaks["hbm"], bound="hbm")
            else:
                row.update(tflops=2.0 * M * N * Kd / us / 1e6, frac=2.0 * M * N * Kd / us / 1e6 / cx.peaks["tf"], bound="tensor")
            out.append(row)
    return out


def _generate(cx, m, vocab, B, P, new, reps):
    prompt = np.random.default_rng(8).integers(0, vocab, size=(B, P)).astype(np.int32)
    m.generate_greedy(prompt, min(8, new))
    pre, dec, steps = [], [], 1
    for _ in range(reps):
        cx.flush_l2()
        cx.sync_all()
        _, t = m.generate_greedy(prompt, new)
        pre.append(t["prefill_ms"]); dec.append(t["decode_ms"]); steps = max(1, t["decode_steps"])
    capi.check_kernel_status(cx.local)
    pre, dec = float(np.median(pre)), float(np.median(dec))
    return dict(batch=B, prompt=P, new=new, prefill_ms=pre, prefill_tokens_per_s=B * P / pre * 1e3, decode_ms_per_step=dec / steps, decode_tokens_per_s=B * steps / dec * 1e3)


def bench_models(cx, reps=3, layers=None):
    from .model import TransformerLM, model_from_config, param_shapes
    work = [(8, 512, 128), (1, 2048, 64), (32, 256, 64)]
    c = model_config()
    if layers:
        c["layers"] = c["layers"][:layers]
    m = model_from_config(c, "bfloat16", max_seq_len=4096)
    rng, n = np.random.default_rng(7), 0
    for name, s in m.param_shapes().items():
        w = 0.02 * rng.standard_normal(s, dtype=np.float32)
        if name.endswith("norm") or name.endswith(("norm1", "norm2", ".D")):
            w += 1.0
        elif name.endswith("dt_bias"):
            w -= 3.0
        m.set_param(name, w)
        n += w.size if name != "bigram" else 0
    hybrid = dict(parameters=n, runs=[_generate(cx, m, c["vocab"], *x, reps) for x in work])
    m.close()
    L = len(c["layers"])
    shapes = param_shapes(32000, 2048, L, 16, 4, 5632)
    t = TransformerLM(32000, 2048, L, 16, 4, 5632, 4096)
    for name, s in shapes.items():
        t.set_param(name, np.ones(s, np.float32) if len(s) == 1 else 0.02 * rng.standard_normal(s, dtype=np.float32))
    llama = dict(parameters=int(sum(np.prod(s) for s in shapes.values())), runs=[_generate(cx, t, 32000, *x, reps) for x in work])
    t.close()
    return dict(hybrid=hybrid, llama_style=llama, layers=L)


def bench_hybrid(cx, K=20, W=3, layers=None, part="all"):
    out = {}
    if part in ("all", "kernels"):
        out["kernels"] = [
            bench_like_prefill(cx, K, W, 4, 2048), bench_like_prefill(cx, K, W, 8, 512), bench_latent_prefill(cx, K, W, 4, 2048, 1 << 20), bench_latent_prefill(cx, K, W, 4, 2048, 1024), bench_latent_prefill(cx, K, W, 8, 512, 1024),
            bench_latent_prefill(cx, K, W, 1, 8192, 1024), bench_latent_prefill(cx, K, W, 2, 2048, 1024, H=64),
            bench_like_decode(cx, K, W, 128, 2304), bench_like_decode(cx, K, W, 32, 2304), bench_like_decode(cx, K, W, 8, 576),       # bytes of the three below
            bench_latent_decode(cx, K, W, 128, 4096), bench_latent_decode(cx, K, W, 32, 4096), bench_latent_decode(cx, K, W, 128, 1024), bench_latent_decode(cx, K, W, 8, 1024), bench_latent_decode(cx, K, W, 32, 4096, H=64),
            bench_ssd(cx, K, W, 8, 512), bench_ssd(cx, K, W, 1, 4096), bench_ssd(cx, K, W, 4, 2048), bench_ssd(cx, K, W, 8, 1), bench_ssd(cx, K, W, 64, 1)]
        out["projections"] = bench_projections(cx, K, W)
    if part in ("all", "models"):
        out["models"] = bench_models(cx, layers=layers)
    return out
