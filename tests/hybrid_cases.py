"""Small hybrid-decoder configurations and seeded weights for the model tests."""
import json
import struct

import numpy as np

from helpers import bf16_round
from hybrid_reference import ReferenceHybrid


def latent(heads, dim, rot_dim, vdim, kv_rank, window, scale=None, base=700.0):
    return dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=kv_rank, scale=scale or (dim + rot_dim) ** -0.5, rot=dict(base=base, dims=rot_dim), mask=dict(size=window))


def mamba(heads, vdim, state, groups, conv, norm_groups):
    return dict(heads=heads, vdim=vdim, state=state, groups=groups, conv=conv, norm_groups=norm_groups)


def layer(mixer, ff=None):
    return dict(type="mamba2" if "state" in mixer else "latent_attention", mixer=mixer, mlp=dict(kind="dense", ff=ff) if ff else None)


def config(vocab, width, layers, loop=None, bigram=None, eps=1e-5):
    c = dict(architecture="Nitenex", vocab=vocab, width=width, norm=dict(eps=eps), layers=layers)
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    if bigram:
        c["embedding"] = dict(bigram=dict(zip(("buckets", "mul_prev", "mul_cur"), bigram)))
    return c


CASES = {
    # a loop inside, layers without feed-forward at both of its ends, an odd vocabulary
    "looped": config(211, 64, [layer(mamba(4, 16, 16, 2, 4, 2), 96), layer(latent(3, 24, 8, 16, 40, 21)), layer(latent(2, 16, 16, 24, 24, 50), 104),
                               layer(mamba(2, 24, 24, 1, 3, 1))], loop=(1, 3, 3), bigram=(89, 13, 5)),
    # nothing is a multiple of 8: width, ff, head sizes, latent
    "ragged": config(130, 100, [layer(latent(3, 10, 6, 12, 33, 9), 60), layer(mamba(5, 7, 10, 5, 2, 5), 61), layer(latent(1, 20, 2, 30, 17, 70), 33)]),
    # one pass over a loop that covers every layer; windows of one and of more than any sequence
    "once": config(96, 72, [layer(latent(4, 16, 8, 16, 32, 1), 80), layer(latent(17, 8, 8, 8, 48, 5000), 80)], loop=(0, 2, 1), bigram=(1, 3, 7)),
    "recurrent": config(64, 48, [layer(mamba(6, 8, 32, 3, 1, 6)), layer(mamba(1, 64, 128, 1, 5, 4), 40)], loop=(0, 1, 2)),
    "tail": config(100, 64, [layer(mamba(4, 32, 40, 4, 4, 1), 64), layer(latent(2, 64, 32, 64, 128, 33), 128), layer(mamba(2, 40, 16, 2, 4, 2))], loop=(1, 2, 2), bigram=(40, 100003, 9)),
}


def shapes(c):
    w, out = c["width"], {"embed": (c["vocab"], c["width"]), "final.norm": (c["width"],)}
    if "embedding" in c:
        out["bigram"] = (c["embedding"]["bigram"]["buckets"] + 1, w)
    if "loop" in c:
        out["loop.step"] = (c["loop"]["times"], w)
    for i, l in enumerate(c["layers"]):
        p, m = f"l{i}.", l["mixer"]
        out[p + "norm1"] = (w,)
        if l["type"] == "latent_attention":
            H, d, r, v, k = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
            sub = {"q": (H * (d + r), w), "dkv": (k + r, w), "dkv.norm": (k,), "uk": (H * d, k), "uv": (H * v, k), "sink": (H,), "o": (w, H * v)}
        else:
            H, inner, gn = m["heads"], m["heads"] * m["vdim"], m["groups"] * m["state"]
            sub = {"in": (2 * inner + 2 * gn + H, w), "conv": (inner + 2 * gn, m["conv"]), "conv.b": (inner + 2 * gn,), "dt_bias": (H,), "A_log": (H,), "D": (H,),
                   "norm": (inner,), "o": (w, inner)}
        out.update({p + "mix." + k: s for k, s in sub.items()})
        if l["mlp"]:
            out.update({p + "norm2": (w,), p + "mlp.up": (l["mlp"]["ff"], w), p + "mlp.down": (w, l["mlp"]["ff"])})
    return out


def weights(c, seed=0):
    """bf16 values; scaled so that every mechanism has a visible share of the residual stream."""
    rng, out = np.random.default_rng(seed), {}
    for name, s in shapes(c).items():
        x = rng.standard_normal(s)
        if name.endswith(("norm", "norm1", "norm2")):
            x = 1 + 0.2 * x
        elif name.endswith("A_log"):
            x = np.log(rng.uniform(0.2, 3.0, s))
        elif name.endswith("dt_bias"):
            x = x - 1.5
        elif name.endswith("mix.conv"):
            x = x / np.sqrt(s[1])
        elif name.endswith("conv.b"):
            x = 0.2 * x
        elif name.endswith((".q", ".dkv")):
            x = 1.6 * x / np.sqrt(s[1])
        elif len(s) == 2 and name not in ("embed", "bigram", "loop.step"):
            x = x / np.sqrt(s[1])
        elif name in ("bigram", "loop.step"):
            x = 0.7 * x
        out[name] = bf16_round(x.astype(np.float32))
    return out


def reference(c, w):
    return ReferenceHybrid(c, w)


def build(c, w, dtype, want_shapes=None, **kw):
    from vesper_b200.model import model_from_config
    m = model_from_config(c, dtype, **kw)
    assert m.param_shapes() == (want_shapes or shapes(c))
    for k, v in w.items():
        m.set_param(k, v)
    return m


def save(folder, c, w):
    """config.json and a bf16 model.safetensors."""
    (folder / "config.json").write_text(json.dumps(c))
    head, data = {"__metadata__": {"format": "pt"}}, b""
    for k, v in w.items():
        raw = (np.ascontiguousarray(v, np.float32).view(np.uint32) >> 16).astype("<u2").tobytes()
        head[k] = dict(dtype="BF16", shape=list(v.shape), data_offsets=[len(data), len(data) + len(raw)])
        data += raw
    h = json.dumps(head).encode()
    (folder / "model.safetensors").write_bytes(struct.pack("<Q", len(h)) + h + data)
