"""Plain NumPy statement of the Zudisun decoder's equations, one function per mechanism, for the tests.

Token by token and head by head where that is the definition; nothing is shared with the product path.  Arithmetic is
float64 unless `real` says otherwise.
"""
import math

import numpy as np

from hybrid_reference import causal_conv, rms_norm, silu, softplus


def sigmoid(x):
    return 0.5 * (1.0 + np.tanh(0.5 * x))


def selective_scan(x, dt, A_log, B, C, D, S):
    """x, dt [T, inner] (dt after softplus), A_log [inner, N], B / C [T, N], S [inner, N]: one token at a time."""
    A = -np.exp(A_log)
    y, S = np.zeros_like(x), S.copy()
    for t in range(x.shape[0]):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        y[t] = S @ C[t] + D * x[t]
    return y, S


def distance_bucket(n, rows, reach):
    """Row of the bias table for a distance n: one row each up to rows/2, then logarithmically up to `reach`."""
    half = rows // 2
    if n < half:
        return n
    if reach <= half:
        return rows - 1
    # an exact power lands on its bucket's edge: nudge the quotient of logarithms past its rounding
    return min(rows - 1, half + int(math.floor(math.log(n / half) / math.log(reach / half) * (rows - half) + 1e-9)))


def query_temperature(p, coef, every):
    return 1.0 + coef * math.log(math.floor((p + 1) / every) + 1.0)


def sigmoid_attention(q, k, v, q_pos, scale, rel, reach, talk, pb):
    """q [T, H, dim], k [L, G, dim], v [L, G, vdim], key j at position j: unnormalised sigmoid weights of mixed scores."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]), q.dtype)
    table = np.array([distance_bucket(n, rel.shape[0], reach) for n in range(int(q_pos[-1]) + 1)])
    for t in range(T):
        n = int(q_pos[t]) + 1
        s = np.stack([(k[:n, h // (H // G)] @ q[t, h]) * scale + rel[table[q_pos[t] - np.arange(n)], h] for h in range(H)])
        w = sigmoid(talk @ s + pb[:, None])
        for h in range(H):
            out[t, h] = w[h] @ v[:n, h // (H // G)]
    return out


def route_margin(logits, correction, top, groups, keep):
    """How far the choice is from another one: the smallest gap between what is taken and what is not, groups and experts."""
    choice, E, gap = sigmoid(logits) + correction, len(logits), np.inf
    if groups:
        score = np.sort(np.sort(choice.reshape(groups, E // groups), axis=1)[:, -2:].sum(axis=1))[::-1]
        if keep < groups:
            gap = score[keep - 1] - score[keep]
    ids, _ = route(logits, correction, E if not groups else keep * (E // groups), groups, keep, 1.0)
    if len(ids) > top:
        gap = min(gap, choice[ids[top - 1]] - choice[ids[top]])
    return gap


def route(logits, correction, top, groups, keep, scale):
    """(expert ids, weights) of one token."""
    s = sigmoid(logits)
    choice = s + correction
    E = len(logits)
    if groups:
        parts = choice.reshape(groups, E // groups)
        score = np.sort(parts, axis=1)[:, -2:].sum(axis=1)
        best = np.argsort(-score, kind="stable")[:keep]
        choice = np.where(np.isin(np.arange(E) // (E // groups), best), choice, -np.inf)
    ids = np.argsort(-choice, kind="stable")[:top]
    return ids, s[ids] / (s[ids].sum() + 1e-20) * scale


class ReferenceZudisun:
    """The whole decoder from a configuration dict (config.json's keys) and a dict of arrays."""

    def __init__(self, config, weights, real=np.float64, round_act=None):
        self.c, self.real = config, real
        self.w = {k: np.asarray(v).astype(real) for k, v in weights.items()}
        self.rnd = round_act if round_act is not None else (lambda a: a)
        self.reset()

    def reset(self):
        self.pos, self.states = 0, {}
        self.margins = {}                  # position -> smallest router margin of its layers

    def lin(self, x, name):
        y = self.rnd(x) @ self.w[name].T
        return self.rnd(y + self.w[name + ".b"] if name + ".b" in self.w else y)

    def mamba1(self, x, i):
        m, p = self.c["layers"][i]["mixer"], f"l{i}.mix."
        inner, N, R = m["inner"], m["state"], m["dt_rank"]
        u = self.lin(x, p + "in")
        w = self.w[p + "conv"]
        before, S = self.states.get(i, (np.zeros((w.shape[1] - 1, inner), self.real), np.zeros((inner, N), self.real)))
        c, before = causal_conv(u[:, :inner], before, w, self.w[p + "conv.b"])
        c = self.rnd(silu(c))
        d = self.lin(c, p + "x")
        dt = softplus(self.rnd(d[:, :R]) @ self.w[p + "dt"].T + self.w[p + "dt.b"])
        y, S = selective_scan(c, dt, self.w[p + "A_log"], d[:, R:R + N], d[:, R + N:], self.w[p + "D"], S)
        self.states[i] = (before, S)
        return self.lin(y * silu(u[:, inner:]), p + "o")

    def attention(self, x, i):
        m, p, eps = self.c["layers"][i]["mixer"], f"l{i}.mix.", self.c["norm"]["eps"]
        H, G, d, dv, T = m["heads"], m["kv_heads"], m["dim"], m["vdim"], x.shape[0]
        pos = np.arange(self.pos, self.pos + T)
        q = rms_norm(self.lin(x, p + "q").reshape(T, H, d), eps)
        k = self.rnd(rms_norm(self.lin(x, p + "k").reshape(T, G, d), eps))
        v = self.lin(x, p + "v").reshape(T, G, dv)
        if m.get("q_temp"):
            q = q * np.array([query_temperature(int(t), m["q_temp"]["coef"], m["q_temp"]["every"]) for t in pos])[:, None, None]
        if m.get("v_mix"):
            if self.v_first is None:
                self.v_first = v
            else:
                lam = float(self.w[p + "vmix"].reshape(()))
                v = self.rnd((1 - lam) * v + lam * self.v_first.reshape(v.shape))
        k0, v0 = self.states.get(i, (np.zeros((0, G, d), self.real), np.zeros((0, G, dv), self.real)))
        k, v = np.concatenate([k0, k]), np.concatenate([v0, v])
        self.states[i] = (k, v)
        o = sigmoid_attention(self.rnd(q), k, v, pos, m["scale"], self.w[p + "rel"], m["bias_max"], self.w[p + "talk"], self.w[p + "pb"])
        o = o * sigmoid(self.lin(x, p + "g"))[:, :, None]
        return self.lin(o.reshape(T, H * dv), p + "o")

    def gated(self, x, name, act):
        return self.lin(act(self.lin(x, name + ".gate")) * self.lin(x, name + ".up"), name + ".down")

    def feed_forward(self, x, i):
        m, p = self.c["layers"][i]["mlp"], f"l{i}.mlp"
        if m["kind"] == "dense":
            return self.gated(x, p, lambda z: np.maximum(z, 0.0))
        r, out = m["router"], np.zeros_like(x)
        logits = self.rnd(x) @ self.w[p + ".router"].T
        g = r.get("groups") or {}
        for t in range(x.shape[0]):
            choice = (logits[t], self.w[p + ".correction"], r["top"], g.get("count"), g.get("keep"))
            ids, weights = route(*choice, r["scale"])
            self.margins[self.pos + t] = min(self.margins.get(self.pos + t, np.inf), route_margin(*choice))
            for e, we in zip(ids, weights):
                out[t] += we * self.gated(x[t:t + 1], f"{p}.e{e}", silu)[0]
        return out + self.gated(x, p + ".shared", silu) if m.get("shared") else out

    def forward(self, tokens, layers_out=None):
        """Logits [T, vocab] of the next tokens of the sequence."""
        w, eps = self.w, self.c["norm"]["eps"]
        tokens = [int(t) for t in tokens]
        x, self.v_first = w["embed"][tokens], None
        for i, L in enumerate(self.c["layers"]):
            x = x + rms_norm(getattr(self, L["type"])(x, i), eps) * w[f"l{i}.norm1"]
            if L.get("mlp"):
                x = x + rms_norm(self.feed_forward(x, i), eps) * w[f"l{i}.norm2"]
            if layers_out is not None:
                layers_out.append(x)
        self.pos += len(tokens)
        return (rms_norm(x, eps) * w["final.norm"]) @ w["head"].T
