"""Plain NumPy statement of the hybrid decoder's equations, one function per mechanism, for the tests.

Everything is written token by token and head by head where that is the definition; nothing is shared with
the product path.  `real` selects the number format of the arithmetic (float64 by default, so that the
checker's own rounding does not matter).
"""
import numpy as np


def rms_norm(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def silu(x):
    return x / (1.0 + np.exp(-x))


def softplus(x):
    return np.logaddexp(0.0, x)


def bigram_rows(tokens, prev, buckets, mul_prev, mul_cur):
    """Table row of every token; prev is None at the start of a sequence (its row is the last one)."""
    rows = []
    for t in tokens:
        rows.append(buckets if prev is None else (int(prev) * mul_prev + int(t) * mul_cur) % buckets)
        prev = t
    return np.array(rows, np.int64)


def rotate_half(x, positions, base, real=np.float64):
    """x [T, ..., R]: all R dimensions rotated, dimension i paired with i + R/2, angle p * base^(-2i/R)."""
    R = x.shape[-1]
    i = np.arange(R // 2, dtype=real)
    f = np.power(real(base), -2.0 * i / R).astype(real)
    a = np.asarray(positions, real)[:, None] * f
    a = a.reshape((len(positions),) + (1,) * (x.ndim - 2) + (R // 2,))
    u, v = x[..., :R // 2], x[..., R // 2:]
    return np.concatenate([u * np.cos(a) - v * np.sin(a), v * np.cos(a) + u * np.sin(a)], axis=-1)


def causal_conv(x, before, w, b):
    """x [T, C]; before [taps - 1, C] inputs ahead of it; w [C, taps], last column = the current token."""
    taps = w.shape[1]
    full = np.concatenate([before, x], axis=0)
    out = np.zeros_like(x)
    for t in range(x.shape[0]):
        out[t] = np.sum(full[t:t + taps] * w.T, axis=0) + b
    return out, full[full.shape[0] - (taps - 1):]


def ssd_scan(x, B, C, dt, A_log, D, state):
    """x [T, H, P], B / C [T, G, N], dt [T, H] (after softplus), state [H, N, P]: the recurrence, one token at a time."""
    T, H, P = x.shape
    G = B.shape[1]
    y = np.zeros_like(x)
    S = state.copy()
    for t in range(T):
        for h in range(H):
            g = h // (H // G)
            S[h] = np.exp(-np.exp(A_log[h]) * dt[t, h]) * S[h] + dt[t, h] * np.outer(B[t, g], x[t, h])
            y[t, h] = S[h].T @ C[t, g] + D[h] * x[t, h]
    return y, S


def gated_group_norm(y, z, w, groups, eps):
    v = y * silu(z)
    parts = v.reshape(v.shape[0], groups, -1)
    return rms_norm(parts, eps).reshape(v.shape) * w


def window_attention_with_sink(q, k, v, q_pos, k_pos, scale, window, sink):
    """q [T, H, Dk], k [L, H, Dk], v [L, H, Dv], sink [H] or None: softmax over visible keys plus the sink."""
    T, H, _ = q.shape
    out = np.zeros((T, H, v.shape[-1]), q.dtype)
    for t in range(T):
        d = q_pos[t] - np.asarray(k_pos)
        vis = (d >= 0) & (d < window)
        for h in range(H):
            s = (k[vis, h] @ q[t, h]) * scale
            m = max(s.max(), sink[h]) if sink is not None else s.max()
            e = np.exp(s - m)
            den = e.sum() + (np.exp(sink[h] - m) if sink is not None else 0.0)
            out[t, h] = (e / den) @ v[vis, h]
    return out


def squared_relu(x):
    return np.square(np.maximum(x, 0.0))


class ReferenceHybrid:
    """The whole decoder from a configuration dict (config.json's keys) and a dict of arrays."""

    def __init__(self, config, weights, real=np.float64, round_act=None):
        self.c, self.real = config, real
        self.w = {k: np.asarray(v).astype(real) for k, v in weights.items()}
        self.rnd = round_act if round_act is not None else (lambda a: a)
        self.reset()

    def reset(self):
        self.pos, self.prev = 0, None
        self.states = {}

    def lin(self, x, name):
        return self.rnd(self.rnd(x) @ self.w[name].T)

    def runs(self):
        """(layer, pass or None, first layer of a pass?) in execution order."""
        n = len(self.c["layers"])
        lp = self.c.get("loop")
        if not lp:
            return [(i, None, False) for i in range(n)]
        out = [(i, None, False) for i in range(lp["start"])]
        for t in range(lp["times"]):
            out += [(i, t, i == lp["start"]) for i in range(lp["start"], lp["stop"])]
        return out + [(i, None, False) for i in range(lp["stop"], n)]

    def latent_attention(self, x, i, key):
        m, p, eps = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.c["norm"]["eps"]
        H, d, r, rank, dv = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"], m["vdim"]
        T = x.shape[0]
        pos = np.arange(self.pos, self.pos + T)
        q = self.lin(x, p + "q").reshape(T, H, d + r)
        q = np.concatenate([q[..., :d], self.rnd(rotate_half(q[..., d:], pos, m["rot"]["base"], self.real))], axis=-1)
        ckv = self.lin(x, p + "dkv")
        c = self.rnd(rms_norm(ckv[:, :rank], eps) * self.w[p + "dkv.norm"])
        kr = self.rnd(rotate_half(ckv[:, None, rank:], pos, m["rot"]["base"], self.real)[:, 0])
        c0, k0 = self.states.get(key, (np.zeros((0, rank), self.real), np.zeros((0, r), self.real)))
        c, kr = np.concatenate([c0, c]), np.concatenate([k0, kr])
        self.states[key] = (c, kr)
        L = c.shape[0]
        lo = max(0, self.pos - m["mask"]["size"] + 1)
        kn = self.lin(c[lo:], p + "uk").reshape(L - lo, H, d)
        v = self.lin(c[lo:], p + "uv").reshape(L - lo, H, dv)
        k = np.concatenate([kn, np.repeat(kr[lo:, None], H, axis=1)], axis=-1)
        o = window_attention_with_sink(q, k, v, pos, np.arange(lo, L), m["scale"], m["mask"]["size"], self.w[p + "sink"])
        return self.lin(o.reshape(T, H * dv), p + "o")

    def mamba2(self, x, i, key):
        m, p, eps = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.c["norm"]["eps"]
        H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
        inner, T = H * P, x.shape[0]
        u = self.lin(x, p + "in")
        z, xbc, dt = u[:, :inner], u[:, inner:2 * inner + 2 * G * N], u[:, 2 * inner + 2 * G * N:]
        w = self.w[p + "conv"]
        before, S = self.states.get(key, (np.zeros((w.shape[1] - 1, w.shape[0]), self.real), np.zeros((H, N, P), self.real)))
        xbc, before = causal_conv(xbc, before, w, self.w[p + "conv.b"])
        xbc = self.rnd(silu(xbc))
        dt = softplus(dt + self.w[p + "dt_bias"])
        y, S = ssd_scan(xbc[:, :inner].reshape(T, H, P), xbc[:, inner:inner + G * N].reshape(T, G, N),
                        xbc[:, inner + G * N:].reshape(T, G, N), dt, self.w[p + "A_log"], self.w[p + "D"], S)
        self.states[key] = (before, S)
        return self.lin(gated_group_norm(y.reshape(T, inner), z, self.w[p + "norm"], m["norm_groups"], eps), p + "o")

    def forward(self, tokens, layers_out=None):
        """Logits [T, vocab] of the next tokens of the sequence."""
        c, w, eps = self.c, self.w, self.c["norm"]["eps"]
        tokens = [int(t) for t in tokens]
        x = w["embed"][tokens]
        bg = c.get("embedding", {}).get("bigram")
        if bg:
            x = x + w["bigram"][bigram_rows(tokens, self.prev, bg["buckets"], bg["mul_prev"], bg["mul_cur"])]
        e = x
        for n, (i, t, first) in enumerate(self.runs()):
            if first:
                if t > 0:
                    x = x + e
                x = x + w["loop.step"][t]
            L = c["layers"][i]
            x = x + getattr(self, L["type"])(rms_norm(x, eps) * w[f"l{i}.norm1"], i, n)
            if L.get("mlp"):
                h = rms_norm(x, eps) * w[f"l{i}.norm2"]
                x = x + self.lin(self.rnd(squared_relu(self.lin(h, f"l{i}.mlp.up"))), f"l{i}.mlp.down")
            if layers_out is not None:
                layers_out.append(x)
        self.pos += len(tokens)
        self.prev = tokens[-1]
        return (rms_norm(x, eps) * w["final.norm"]) @ w["embed"].T
