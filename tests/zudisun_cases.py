"""Small Zudisun configurations and seeded weights for the model tests."""
import numpy as np

import hybrid_cases
from helpers import bf16_round
from hybrid_cases import save      # noqa: F401
from zudisun_reference import ReferenceZudisun


def attention(heads, kv_heads, dim, vdim, rel, bias_max, scale=None, temp=None, v_mix=True):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale or dim ** -0.5, bias_max=bias_max, rel=rel)
    if temp:
        m["q_temp"] = dict(coef=temp[0], every=temp[1])
    if v_mix is not None:
        m["v_mix"] = v_mix
    return m


def mamba(inner, state, dt_rank, conv):
    return dict(inner=inner, state=state, dt_rank=dt_rank, conv=conv)


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(ff, experts, top, scale, groups=None, shared=None):
    m = dict(kind="moe", expert=dict(ff=ff), router=dict(experts=experts, top=top, scale=scale))
    if groups:
        m["router"]["groups"] = dict(count=groups[0], keep=groups[1])
    if shared:
        m["shared"] = dict(ff=shared)
    return m


def config(vocab, width, layers, eps=1e-5):
    """layers: (mixer, feed-forward or None).  The rows of a bias table are no key of the configuration: the table's shape gives them."""
    out, rel = [], []
    for mixer, mlp in layers:
        mixer = dict(mixer)
        rel.append(mixer.pop("rel", None))
        out.append(dict(type="mamba1" if "inner" in mixer else "attention", mixer=mixer, mlp=mlp))
    return dict(architecture="Zudisun", vocab=vocab, width=width, norm=dict(eps=eps), layers=out), rel


CASES = {
    # attention first and last, Mamba between, value mixing over a gap; heads in groups of three; a sharp temperature
    "mixed": config(150, 96, [(attention(6, 2, 24, 16, 12, 50, temp=(0.6, 20)), dense(80)), (mamba(72, 16, 8, 4), moe(40, 6, 2, 1.7, groups=(3, 2), shared=48)),
                              (attention(4, 4, 32, 8, 8, 33, temp=(0.2, 7)), moe(24, 12, 5, 0.9)), (mamba(40, 40, 20, 3), None),
                              (attention(8, 2, 16, 16, 20, 100, scale=0.4), dense(64))]),
    # nothing is a multiple of 8
    "ragged": config(133, 52, [(mamba(44, 10, 5, 2), dense(31)), (attention(3, 3, 10, 12, 6, 9.5, temp=(1.3, 3), v_mix=False), moe(19, 5, 1, 2.0, shared=13)),
                               (attention(6, 2, 14, 18, 10, 40), None), (mamba(30, 3, 1, 1), moe(21, 4, 4, 1.1, groups=(2, 2), shared=5)), (attention(2, 2, 6, 18, 2, 3), dense(50))]),
    # Mamba only, a state wider than the kernels' smallest shapes; a layer with one expert
    "recurrent": config(64, 48, [(mamba(64, 72, 24, 4), moe(32, 1, 1, 1.0, shared=16)), (mamba(16, 136, 3, 5), None)]),
    # wide heads: the tensor-core kernels at their limits, many experts in groups of one
    "wide": config(96, 128, [(attention(16, 4, 128, 128, 32, 64, scale=0.09, temp=(0.4, 32)), moe(64, 32, 6, 2.5, groups=(8, 3), shared=96)),
                             (attention(16, 4, 128, 128, 18, 200, scale=0.11), moe(48, 10, 3, 1.0, groups=(10, 4)))]),
}


def case(name):
    """(configuration, rows of every layer's bias table)"""
    return CASES[name]


def shapes(c, rel):
    """Parameter shapes; rel: rows of the layers' bias tables."""
    w, out = c["width"], {"embed": (c["vocab"], c["width"]), "head": (c["vocab"], c["width"]), "final.norm": (c["width"],)}
    mixing = [i for i, l in enumerate(c["layers"]) if l["mixer"].get("v_mix")]
    for i, l in enumerate(c["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = (w,)
        if l["type"] == "attention":
            H, G, d, v = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            sub = {"q": (H * d, w), "k": (G * d, w), "v": (G * v, w), "g": (H, w), "rel": (rel[i], H), "talk": (H, H), "pb": (H,), "o": (w, H * v)}
            if i in mixing:
                sub["vmix"] = ()
        else:
            n, s, r = m["inner"], m["state"], m["dt_rank"]
            sub = {"in": (2 * n, w), "conv": (n, m["conv"]), "conv.b": (n,), "x": (r + 2 * s, n), "dt": (n, r), "dt.b": (n,), "A_log": (n, s), "D": (n,), "o": (w, n)}
        out.update({p + "mix." + k: s for k, s in sub.items()})
        mlp = l["mlp"]
        if not mlp:
            continue
        out[p + "norm2"] = (w,)

        def gated(q, ff):
            out.update({q + ".gate": (ff, w), q + ".up": (ff, w), q + ".down": (w, ff)})
        if mlp["kind"] == "dense":
            gated(p + "mlp", mlp["ff"])
            out.update({p + "mlp.gate.b": (mlp["ff"],), p + "mlp.up.b": (mlp["ff"],), p + "mlp.down.b": (w,)})
        else:
            E = mlp["router"]["experts"]
            out.update({p + "mlp.router": (E, w), p + "mlp.correction": (E,)})
            for e in range(E):
                gated(f"{p}mlp.e{e}", mlp["expert"]["ff"])
            if mlp.get("shared"):
                gated(p + "mlp.shared", mlp["shared"]["ff"])
    return out


def weights(c, rel, seed=0):
    """bf16 values; scaled so that every mechanism has a visible share of the residual stream, and no router call is close."""
    rng, out = np.random.default_rng(seed), {}
    for name, s in shapes(c, rel).items():
        x = rng.standard_normal(s)
        last = name.rsplit(".", 1)[-1]
        if last in ("norm", "norm1", "norm2"):
            x = 1 + 0.2 * x
        elif last == "A_log":
            x = np.log(rng.uniform(0.02, 4.0, s))
        elif name.endswith("dt.b"):
            x = x - 2.0
        elif last == "conv":
            x = x / np.sqrt(s[1])
        elif last == "b":
            x = 0.3 * x
        elif last == "rel":
            x = 1.5 * x
        elif last == "pb":
            x = 0.5 * x - 3.0
        elif last == "talk":
            x = np.eye(s[0]) + 0.4 * x / np.sqrt(s[0])
        elif last == "vmix":
            x = np.asarray(0.3)
        elif last == "correction":
            x = 0.5 * x - 1.5
        elif last in ("q", "k"):
            x = 1.6 * x / np.sqrt(s[1])
        elif last == "router":
            x = 2.0 * x / np.sqrt(s[1])
        elif len(s) == 2 and name != "embed":
            x = x / np.sqrt(s[1])
        out[name] = bf16_round(np.asarray(x, np.float32)).reshape(s)
    return out


def build(c, rel, w, dtype, **kw):
    want = {k: (-1,) + s[1:] if k.endswith("mix.rel") else s for k, s in shapes(c, rel).items()}
    return hybrid_cases.build(c, w, dtype, want_shapes=want, **kw)


def reference(c, w, **kw):
    return ReferenceZudisun(c, w, **kw)
