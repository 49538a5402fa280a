"""Logits of a model under test against the plain model, position by position.

The error at a position is the rms over the vocabulary of the logit difference, relative to the rms of all logits of
the case.  Limit in fp32: 1e-4.  In bf16: three times what rounding alone does there, taken from runs of the plain model
with every activation rounded to bf16 at a random place within half a step (random small models have ill-conditioned
positions; a window, key, tap or state that is wrong costs far more).  Positions where a router's choice is close are left out in
bf16, with the two after them: rounding may pick another expert there."""
import numpy as np

from helpers import bf16_round


def errors(got, want):
    d = got - want
    return np.sqrt((d * d).mean(-1)) / np.sqrt((want * want).mean())


class Sequence:
    """Token ids with the plain model's logits and the error limit at every position.  plain(config, weights, round_act=...) makes the
    plain model."""

    def __init__(self, plain, c, w, ids, trials=5):
        model = plain(c, w)
        self.ids, self.want = ids, model.forward(ids)
        margins = getattr(model, "margins", {})
        margin = np.array([margins.get(t, np.inf) for t in range(len(ids))])
        close = margin < 0.02
        for n in (1, 2):                                 # what another expert changes there reaches the next tokens through their convolutions
            close[n:] |= margin[:-n] < 0.01
        assert close.mean() < 0.6
        self.skip = {"float32": np.zeros(len(ids), bool), "bfloat16": close}
        rng = np.random.default_rng(11)

        def dither(a):
            a = a.astype(np.float32)
            return bf16_round(a * (1 + (rng.random(a.shape).astype(np.float32) - 0.5) * 2 ** -8)).astype(np.float64)
        e = np.max([errors(plain(c, w, round_act=dither).forward(ids), self.want) for _ in range(trials)], axis=0)
        self.limits = {"float32": np.full(len(ids), 1e-4), "bfloat16": 3 * np.maximum(e, np.quantile(e, 0.9))}
        self.rms = np.sqrt((self.want ** 2).mean())

    def check(self, got, dtype, at=0, scale=1.0):
        n = len(got)
        d = got - self.want[at:at + n]
        over = np.sqrt((d * d).mean(-1)) / self.rms / self.limits[dtype][at:at + n]
        over = np.where(self.skip[dtype][at:at + n], 0.0, over)
        assert over.max() <= scale, (at + int(over.argmax()), over.max())


def run(m, ids, cuts):
    """A sequence of its own through the model in portions; logits of every token."""
    s = m.open_sequence()
    out, at = [], 0
    for n in cuts:
        out.append(m.extend(s, ids[at:at + n]))
        at += n
    m.close_sequence(s)
    status()
    return np.concatenate(out)


def status():
    from vesper_b200 import capi
    capi.check_kernel_status(0)
