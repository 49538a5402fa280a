"""ctypes binding of include/vesper_b200_hybrid.h for the tests and the benchmark, on torch tensors: the operators of
hybrid decoders, and the cores of the sequence mixers with their cache or state around them."""
from __future__ import annotations

import ctypes as C

from . import capi

HYBRID_EXPORTS = ["vb200_embed_sequence", "vb200_residual_add", "vb200_rms_norm_f32", "vb200_linear_f32_ex", "vb200_latent_workspace_bytes",
                  "vb200_latent_append", "vb200_latent_prefill", "vb200_latent_decode", "vb200_last_latent_kernel", "vb200_ssd_workspace_bytes",
                  "vb200_ssd_forward", "vb200_last_ssd_kernel", "vb200_norm_add", "vb200_sigattn_workspace_bytes", "vb200_sigattn_forward", "vb200_last_sigattn_kernel",
                  "vb200_selective_workspace_bytes", "vb200_selective_forward", "vb200_last_selective_kernel", "vb200_moe_workspace_bytes", "vb200_moe_forward",
                  "vb200_moe_rows", "vb200_moe_rows_of", "vb200_moe_route", "vb200_last_moe_kernel"]

_i32, _i64, _p, _f = C.c_int32, C.c_int64, C.c_void_p, C.c_float


class EmbedArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("dtype", _i32), ("ids", _p), ("B", _i32), ("T", _i32), ("dim", _i32),
                ("vocab", _i32), ("table", _p), ("bigram", _p), ("buckets", _i64), ("mul_prev", _i64), ("mul_cur", _i64), ("slots", _p), ("lens", _p),
                ("step_pos", _p), ("prev", _p), ("h", _p), ("embed_copy", _p), ("add", _p), ("scale", _p), ("scaled_out", _p)]


class LatentArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("dtype", _i32), ("B", _i32), ("T", _i32), ("H", _i32), ("dim", _i32),
                ("rot_dim", _i32), ("vdim", _i32), ("rank", _i32), ("window", _i32), ("ring", _i32), ("scale", _f), ("eps", _f), ("inv_freq", _p),
                ("proj", _p), ("ldp", _i64), ("c_norm", _p), ("w_uk", _p), ("w_uv", _p), ("ldu", _i64), ("sink", _p), ("slots", _p), ("pos", _p),
                ("cache", _p), ("ldc", _i64), ("out", _p), ("ldo", _i64), ("start_pos", _i32), ("ctx_latent", _p), ("ctx_kv", _p), ("ldkv", _i64),
                ("max_len", _i32), ("workspace", _p), ("workspace_bytes", C.c_size_t)]


class SsdArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("dtype", _i32), ("B", _i32), ("T", _i32), ("H", _i32), ("P", _i32),
                ("N", _i32), ("G", _i32), ("taps", _i32), ("norm_groups", _i32), ("eps", _f), ("proj", _p), ("ldp", _i64), ("conv_w", _p), ("conv_b", _p),
                ("dt_bias", _p), ("A_log", _p), ("D", _p), ("norm_w", _p), ("slots", _p), ("pos", _p), ("conv_state", _p), ("state", _p), ("out", _p),
                ("ldo", _i64), ("workspace", _p), ("workspace_bytes", C.c_size_t), ("form", _i32)]



class NormAddArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("M", _i32), ("dim", _i32), ("count", _i32), ("eps", _f), ("x", _p), ("y", _p), ("w", _p),
                ("rows", _p), ("gather", _p), ("n_gather", _i32), ("scale", _p), ("copy_out", _p)]


class SigattnArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("dtype", _i32), ("B", _i32), ("T", _i32), ("H", _i32), ("G", _i32), ("dim", _i32),
                ("vdim", _i32), ("scale", _f), ("eps", _f), ("temp_coef", _f), ("temp_every", _i32), ("proj", _p), ("ldp", _i64), ("talk", _p), ("bias", _p), ("n_bias", _i32),
                ("value_role", _i32), ("lambda_", _f), ("first_values", _p), ("slots", _p), ("pos", _p), ("k_cache", _p), ("ldk", _i64), ("v_cache", _p), ("ldv", _i64),
                ("cap", _i32), ("out", _p), ("ldo", _i64), ("start_pos", _i32), ("max_len", _i32), ("workspace", _p), ("workspace_bytes", C.c_size_t), ("form", _i32)]


class SelectiveArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("dtype", _i32), ("B", _i32), ("T", _i32), ("inner", _i32), ("N", _i32), ("rank", _i32),
                ("taps", _i32), ("proj", _p), ("ldp", _i64), ("conv_w", _p), ("conv_b", _p), ("w_x", _p), ("w_dt", _p), ("dt_bias", _p), ("A", _p), ("D", _p), ("slots", _p),
                ("pos", _p), ("conv_state", _p), ("state", _p), ("out", _p), ("ldo", _i64), ("workspace", _p), ("workspace_bytes", C.c_size_t)]


class MoeArgs(C.Structure):
    _fields_ = [("struct_size", C.c_size_t), ("device", _i32), ("stream", _p), ("dtype", _i32), ("M", _i32), ("dim", _i32), ("ff", _i32), ("ff_shared", _i32), ("experts", _i32),
                ("top", _i32), ("groups", _i32), ("keep", _i32), ("scale", _f), ("x", _p), ("w_router", _p), ("correction", _p), ("w_in", _p), ("w_out", _p), ("ld_out", _i64),
                ("w_shared_in", _p), ("w_shared_out", _p), ("ld_shared", _i64), ("y", _p), ("workspace", _p), ("workspace_bytes", C.c_size_t), ("form", _i32)]


_lib = None


def load():
    global _lib
    if _lib is None:
        L = capi.load()
        for name in ("vb200_latent_workspace_bytes", "vb200_latent_append", "vb200_latent_prefill", "vb200_latent_decode"):
            getattr(L, name).argtypes = [C.POINTER(LatentArgs)]
        for name in ("vb200_ssd_workspace_bytes", "vb200_ssd_forward"):
            getattr(L, name).argtypes = [C.POINTER(SsdArgs)]
        L.vb200_latent_workspace_bytes.restype = C.c_size_t
        L.vb200_ssd_workspace_bytes.restype = C.c_size_t
        L.vb200_embed_sequence.argtypes = [C.POINTER(EmbedArgs)]
        L.vb200_residual_add.argtypes = [C.c_int, _p, _p, _p, _p, _i32, _i32, _p, _p]
        L.vb200_rms_norm_f32.argtypes = [C.c_int, _p, _p, _p, _p, _i32, _i32, _i32, _f]
        L.vb200_linear_f32_ex.argtypes = [C.c_int, _p, _p, _i64, _p, _i64, _p, _p, _p, _i64, _i32, _i32, _i32, _i32]
        for name, args in (("sigattn", SigattnArgs), ("selective", SelectiveArgs), ("moe", MoeArgs)):
            getattr(L, f"vb200_{name}_workspace_bytes").argtypes = getattr(L, f"vb200_{name}_forward").argtypes = [C.POINTER(args)]
            getattr(L, f"vb200_{name}_workspace_bytes").restype = C.c_size_t
            getattr(L, f"vb200_last_{name}_kernel").restype = C.c_char_p
        L.vb200_norm_add.argtypes = [C.POINTER(NormAddArgs)]
        L.vb200_moe_rows.argtypes = [C.POINTER(MoeArgs)]
        L.vb200_moe_rows_of.argtypes = [C.POINTER(MoeArgs), C.POINTER(_p), C.POINTER(_p)]
        L.vb200_moe_route.argtypes = [C.c_int, _p, _p, _p, _i32, _i32, _i32, _i32, _i32, _f, _p, _p]
        L.vb200_last_latent_kernel.restype = C.c_char_p
        L.vb200_last_ssd_kernel.restype = C.c_char_p
        _lib = L
    return _lib


def _pad8(n):
    return (n + 7) // 8 * 8


def _ptr(t):
    return None if t is None else t.data_ptr()


def _stream():
    import torch
    return torch.cuda.current_stream().cuda_stream


def embed_sequence(ids, table, lens, prev, *, bigram=None, buckets=0, mul_prev=0, mul_cur=0, slots=None, add=None, scale=None, want_copy=False):
    """Returns (h [B*T, dim] fp32, embedding copy or None, scaled bf16 copy or None, step_pos)."""
    import torch
    B, T = ids.shape
    dim = table.shape[1]
    h = torch.empty(B * T, dim, device=ids.device)
    e = torch.empty_like(h) if want_copy else None
    xs = torch.empty(B * T, dim, dtype=torch.bfloat16, device=ids.device) if scale is not None else None
    step = torch.empty(B, dtype=torch.int32, device=ids.device)
    a = EmbedArgs(struct_size=C.sizeof(EmbedArgs), stream=_stream(), dtype=capi.dtype_code(table), ids=_ptr(ids), B=B, T=T, dim=dim, vocab=table.shape[0],
                  table=_ptr(table), bigram=_ptr(bigram), buckets=buckets, mul_prev=mul_prev, mul_cur=mul_cur, slots=_ptr(slots), lens=_ptr(lens),
                  step_pos=_ptr(step), prev=_ptr(prev), h=_ptr(h), embed_copy=_ptr(e), add=_ptr(add), scale=_ptr(scale), scaled_out=_ptr(xs))
    capi.check(load().vb200_embed_sequence(C.byref(a)))
    return h, e, xs, step


class LatentCore:
    """Latent attention between its projections: weights [W_uk; W_uv] (rows padded to 8 columns), c_norm, sink, and the ring of `slots` sequences."""

    def __init__(self, *, H, dim, rot_dim, vdim, rank, window, scale, eps, inv_freq, expand, c_norm, sink, slots, max_len=None, dtype=None):
        import torch
        dev = expand.device
        self.dtype = dtype or expand.dtype
        self.s = dict(H=H, dim=dim, rot_dim=rot_dim, vdim=vdim, rank=rank, window=window, ring=min(window, max_len or window))
        self.scale, self.eps, self.sink = scale, eps, sink
        self.inv_freq = torch.as_tensor(inv_freq, dtype=torch.float64, device=dev)
        self.expand = torch.zeros(H * (dim + vdim), _pad8(rank), dtype=self.dtype, device=dev)
        self.expand[:, :rank] = expand
        self.c_norm = c_norm
        self.ldc = _pad8(rank) + _pad8(rot_dim)
        self.cache = torch.zeros(slots, self.s["ring"], self.ldc, dtype=self.dtype, device=dev)
        self.proj_cols = H * (dim + rot_dim) + rank + rot_dim

    def proj_buffer(self, rows):
        import torch
        return torch.zeros(rows, _pad8(self.proj_cols), dtype=self.dtype, device=self.cache.device)

    def _args(self, proj, B, T, pos, slots):
        import torch
        out = torch.zeros(B * T, _pad8(self.s["H"] * self.s["vdim"]), dtype=self.dtype, device=proj.device)
        a = LatentArgs(struct_size=C.sizeof(LatentArgs), stream=_stream(), dtype=capi.dtype_code(proj), B=B, T=T, scale=self.scale, eps=self.eps,
                       inv_freq=_ptr(self.inv_freq), proj=_ptr(proj), ldp=proj.stride(0), c_norm=_ptr(self.c_norm), w_uk=_ptr(self.expand),
                       w_uv=_ptr(self.expand[self.s["H"] * self.s["dim"]:]), ldu=self.expand.stride(0), sink=_ptr(self.sink), slots=_ptr(slots), pos=_ptr(pos),
                       cache=_ptr(self.cache), ldc=self.ldc, out=_ptr(out), ldo=out.stride(0), **self.s)
        return a, out

    def prefill(self, proj, B, start_pos, pos=None, slots=None):
        """proj [B*T, >= proj_cols] (q is rotated in place); all rows start at start_pos.  Returns [B*T, H*vdim]."""
        import torch
        T = proj.shape[0] // B
        dev = proj.device
        pos = pos if pos is not None else torch.full((B,), start_pos, dtype=torch.int32, device=dev)
        a, out = self._args(proj, B, T, pos, slots)
        n = min(start_pos, self.s["window"] - 1) + T
        lat = torch.empty(B * n, self.ldc, dtype=self.dtype, device=dev).fill_(float("nan"))
        N = self.expand.shape[0]
        kv = torch.empty(B * n, _pad8(N), dtype=self.dtype, device=dev)
        a.start_pos, a.ctx_latent, a.ctx_kv, a.ldkv = start_pos, _ptr(lat), _ptr(kv), kv.stride(0)
        L = load()
        capi.check(L.vb200_latent_append(C.byref(a)))
        if self.dtype == torch.float32:
            capi.check(L.vb200_linear_f32(0, _stream(), _ptr(lat), self.ldc, _ptr(self.expand), self.expand.stride(0), None, _ptr(kv), kv.stride(0), B * n, N, self.s["rank"]))
        else:
            capi.check(L.vb200_linear(0, _stream(), _ptr(lat), self.ldc, _ptr(self.expand), self.expand.stride(0), _ptr(kv), kv.stride(0), B * n, N,
                                      self.expand.stride(0), capi.EPI_BF16, 0))
        capi.check(L.vb200_latent_prefill(C.byref(a)))
        self._keep = (lat, kv, pos)
        return out[:, :self.s["H"] * self.s["vdim"]]

    def decode(self, proj, pos, slots=None, max_len=0):
        import torch
        B = proj.shape[0]
        a, out = self._args(proj, B, 1, pos, slots)
        a.max_len = max_len
        a.workspace_bytes = load().vb200_latent_workspace_bytes(C.byref(a))
        ws = torch.empty(a.workspace_bytes // 4, device=proj.device)
        a.workspace = _ptr(ws)
        capi.check(load().vb200_latent_decode(C.byref(a)))
        self._keep = (ws,)
        return out[:, :self.s["H"] * self.s["vdim"]]

    @staticmethod
    def last_kernel():
        return load().vb200_last_latent_kernel().decode()


class SsdCore:
    """The Mamba-2 mixer between its projections, with the convolution ring and state of `slots` sequences."""

    def __init__(self, *, H, P, N, G, taps, norm_groups, eps, conv_w, conv_b, dt_bias, A_log, D, norm_w, slots, dtype):
        import torch
        dev = conv_w.device
        self.dtype = dtype
        self.s = dict(H=H, P=P, N=N, G=G, taps=taps, norm_groups=norm_groups, eps=eps)
        self.w = dict(conv_w=conv_w.contiguous(), conv_b=conv_b, dt_bias=dt_bias, A_log=A_log, D=D, norm_w=norm_w)
        ch = H * P + 2 * G * N
        self.conv_state = torch.zeros(slots, taps, ch, dtype=dtype, device=dev)
        self.state = torch.zeros(slots, H, N, (P + 3) // 4 * 4, device=dev)
        self.proj_cols = 2 * H * P + 2 * G * N + H

    def proj_buffer(self, rows):
        import torch
        return torch.zeros(rows, _pad8(self.proj_cols), dtype=self.dtype, device=self.state.device)

    def forward(self, proj, B, pos, slots=None, form=0):
        import torch
        T = proj.shape[0] // B
        inner = self.s["H"] * self.s["P"]
        out = torch.zeros(B * T, _pad8(inner), dtype=self.dtype, device=proj.device)
        a = SsdArgs(struct_size=C.sizeof(SsdArgs), stream=_stream(), dtype=capi.dtype_code(proj), B=B, T=T, proj=_ptr(proj), ldp=proj.stride(0), slots=_ptr(slots),
                    pos=_ptr(pos), conv_state=_ptr(self.conv_state), state=_ptr(self.state), out=_ptr(out), ldo=out.stride(0), form=form, **self.s,
                    **{k: _ptr(v) for k, v in self.w.items()})
        a.workspace_bytes = load().vb200_ssd_workspace_bytes(C.byref(a))
        ws = torch.empty(a.workspace_bytes // 4 + 1, device=proj.device)
        a.workspace = _ptr(ws)
        capi.check(load().vb200_ssd_forward(C.byref(a)))
        self._keep = (ws,)
        return out[:, :inner]

    @staticmethod
    def last_kernel():
        return load().vb200_last_ssd_kernel().decode()


def norm_add(x, y, w, eps, *, count=None, rows=None, gather=None, scale=None, copy=False):
    """x [M, dim] fp32 in place; returns the bf16 copy (or None)."""
    import torch
    M, dim = x.shape
    out = torch.empty(M, dim, dtype=torch.bfloat16, device=x.device) if copy else None
    a = NormAddArgs(struct_size=C.sizeof(NormAddArgs), stream=_stream(), M=M, dim=dim, count=count or dim, eps=eps, x=_ptr(x), y=_ptr(y), w=_ptr(w), rows=_ptr(rows),
                    gather=_ptr(gather), n_gather=0 if gather is None else gather.shape[1], scale=_ptr(scale), copy_out=_ptr(out))
    capi.check(load().vb200_norm_add(C.byref(a)))
    return out


class SigmoidCore:
    """Sigmoid attention with mixed heads between its projections, with the cache of `slots` sequences.  talk [H, H], bias [H, distances]."""

    def __init__(self, *, H, G, dim, vdim, scale, eps, talk, bias, slots, cap, dtype, temp_coef=0.0, temp_every=0):
        import torch
        dev = talk.device
        self.dtype = dtype
        self.s = dict(H=H, G=G, dim=dim, vdim=vdim, scale=scale, eps=eps, temp_coef=temp_coef, temp_every=temp_every, n_bias=bias.shape[1], cap=cap)
        self.talk, self.bias = talk.float().contiguous(), bias.float().contiguous()
        self.k_cache = torch.zeros(slots, cap, _pad8(G * dim), dtype=dtype, device=dev)
        self.v_cache = torch.zeros(slots, cap, _pad8(G * vdim), dtype=dtype, device=dev)
        self.proj_cols = H * (dim + 1) + G * (dim + vdim)

    def proj_buffer(self, rows):
        import torch
        return torch.zeros(rows, _pad8(self.proj_cols), dtype=self.dtype, device=self.talk.device)

    def forward(self, proj, B, start_pos, pos=None, slots=None, form=0, max_len=0, value_role=0, lam=0.0, first_values=None):
        """proj [B*T, >= proj_cols]; all rows at start_pos when T > 1.  Returns [B*T, H*vdim]."""
        import torch
        T, s = proj.shape[0] // B, self.s
        if pos is None:
            pos = torch.full((B,), start_pos, dtype=torch.int32, device=proj.device)
        out = torch.zeros(B * T, _pad8(s["H"] * s["vdim"]), dtype=self.dtype, device=proj.device)
        a = SigattnArgs(struct_size=C.sizeof(SigattnArgs), stream=_stream(), dtype=capi.dtype_code(proj), B=B, T=T, proj=_ptr(proj), ldp=proj.stride(0), talk=_ptr(self.talk),
                        bias=_ptr(self.bias), value_role=value_role, lambda_=lam, first_values=_ptr(first_values), slots=_ptr(slots), pos=_ptr(pos), k_cache=_ptr(self.k_cache),
                        ldk=self.k_cache.stride(1), v_cache=_ptr(self.v_cache), ldv=self.v_cache.stride(1), out=_ptr(out), ldo=out.stride(0), start_pos=start_pos, max_len=max_len,
                        form=form, **s)
        a.workspace_bytes = load().vb200_sigattn_workspace_bytes(C.byref(a))
        ws = torch.empty(a.workspace_bytes // 4 + 1, device=proj.device)
        a.workspace = _ptr(ws)
        capi.check(load().vb200_sigattn_forward(C.byref(a)))
        self._keep = (ws, pos)
        return out[:, :s["H"] * s["vdim"]]

    @staticmethod
    def last_kernel():
        return load().vb200_last_sigattn_kernel().decode()


class SelectiveCore:
    """The per-channel selective state-space mixer between its projections.  Sizes are multiples of 8; A [inner, N] is negative."""

    def __init__(self, *, inner, N, rank, taps, conv_w, conv_b, w_x, w_dt, dt_bias, A, D, slots, dtype):
        import torch
        dev = A.device
        self.dtype = dtype
        self.s = dict(inner=inner, N=N, rank=rank, taps=taps)
        self.w = dict(conv_w=conv_w.contiguous(), conv_b=conv_b, w_x=w_x.to(dtype).contiguous(), w_dt=w_dt.to(dtype).contiguous(), dt_bias=dt_bias, A=A.contiguous(), D=D)
        self.conv_state = torch.zeros(slots, taps, inner, dtype=dtype, device=dev)
        self.state = torch.zeros(slots, inner, N, device=dev)

    def forward(self, proj, B, pos, slots=None):
        """proj [B*T, >= 2 * inner]: x | z.  Returns [B*T, inner]."""
        import torch
        T = proj.shape[0] // B
        out = torch.zeros(B * T, self.s["inner"], dtype=self.dtype, device=proj.device)
        a = SelectiveArgs(struct_size=C.sizeof(SelectiveArgs), stream=_stream(), dtype=capi.dtype_code(proj), B=B, T=T, proj=_ptr(proj), ldp=proj.stride(0), slots=_ptr(slots),
                          pos=_ptr(pos), conv_state=_ptr(self.conv_state), state=_ptr(self.state), out=_ptr(out), ldo=out.stride(0), **self.s,
                          **{k: _ptr(v) for k, v in self.w.items()})
        a.workspace_bytes = load().vb200_selective_workspace_bytes(C.byref(a))
        ws = torch.empty(a.workspace_bytes // 4 + 1, device=proj.device)
        a.workspace = _ptr(ws)
        capi.check(load().vb200_selective_forward(C.byref(a)))
        self._keep = (ws, pos)
        return out

    @staticmethod
    def last_kernel():
        return load().vb200_last_selective_kernel().decode()


def moe_route(logits, correction, top, groups, keep, scale):
    """(ids, weights) [M, top]."""
    import torch
    M, E = logits.shape
    ids = torch.empty(M, top, dtype=torch.int32, device=logits.device)
    w = torch.empty(M, top, device=logits.device)
    capi.check(load().vb200_moe_route(0, _stream(), _ptr(logits), _ptr(correction), M, E, top, groups, keep, scale, _ptr(ids), _ptr(w)))
    return ids, w


class MoeCore:
    """A mixture of experts: w_gate / w_up [E, ff, dim], w_down [E, dim, ff], shared (gate, up, down) or None; stored as the kernels want them."""

    def __init__(self, *, router, correction, gate, up, down, shared, top, groups, keep, scale, dtype):
        import torch
        self.dtype = dtype

        def mix(g, u):                                   # gate and up rows interleaved
            return torch.stack([g, u], dim=-2).flatten(-3, -2).to(dtype).contiguous()

        def pad(d):
            out = torch.zeros(*d.shape[:-1], _pad8(d.shape[-1]), dtype=dtype, device=d.device)
            out[..., :d.shape[-1]] = d
            return out
        E, ff, dim = gate.shape
        self.router, self.correction = router.to(dtype).contiguous(), correction
        self.w_in, self.w_out = mix(gate, up), pad(down)
        self.shared = (mix(shared[0], shared[1]), pad(shared[2])) if shared else None
        self.s = dict(dim=dim, ff=ff, ff_shared=shared[0].shape[0] if shared else 0, experts=E, top=top, groups=groups, keep=keep, scale=scale)

    def forward(self, x, form=0):
        """(y [M, dim] fp32, rows bf16 or None, gather or None): the output is y plus the gathered rows."""
        import torch
        M = x.shape[0]
        y = torch.empty(M, x.shape[1], device=x.device).fill_(float("nan"))
        a = MoeArgs(struct_size=C.sizeof(MoeArgs), stream=_stream(), dtype=capi.dtype_code(x), M=M, x=_ptr(x), w_router=_ptr(self.router), correction=_ptr(self.correction),
                    w_in=_ptr(self.w_in), w_out=_ptr(self.w_out), ld_out=self.w_out.shape[-1], y=_ptr(y), form=form, **self.s)
        if self.shared:
            a.w_shared_in, a.w_shared_out, a.ld_shared = _ptr(self.shared[0]), _ptr(self.shared[1]), self.shared[1].shape[-1]
        L = load()
        a.workspace_bytes = L.vb200_moe_workspace_bytes(C.byref(a))
        ws = torch.empty(a.workspace_bytes, dtype=torch.uint8, device=x.device)
        a.workspace = _ptr(ws)
        capi.check(L.vb200_moe_forward(C.byref(a)))
        self._keep = ws
        n = L.vb200_moe_rows(C.byref(a))
        if n == 0:
            return y, None, None
        rows, gather = _p(), _p()
        capi.check(L.vb200_moe_rows_of(C.byref(a), C.byref(rows), C.byref(gather)))
        r0, g0 = rows.value - ws.data_ptr(), gather.value - ws.data_ptr()
        pairs = M * n
        return (y, ws[r0:r0 + pairs * x.shape[1] * 2].view(torch.bfloat16).view(pairs, -1), ws[g0:g0 + pairs * 4].view(torch.int32).view(M, n))

    @staticmethod
    def last_kernel():
        return load().vb200_last_moe_kernel().decode()
