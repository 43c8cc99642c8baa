"""Small layered models for the tests, and running them on the device and in the plain restatement."""
import numpy as np

import lm_oracle


def variants(synth):
    """name -> configuration. Sizes are chosen so that no two of them coincide by accident."""
    L = synth.layered_layer
    return {
        # grouped heads, two windows, a layer without feed-forward, shared weights with another layer between
        "mixed": synth.layered_config(211, 144, [L(6, 3, 24, 40, 19, 200, coef=0.4, every=7), L(4, 1, 32, 16, 70, None, coef=0.1, every=33),
                                                 L(6, 3, 24, 40, 19, 200, coef=0.4, every=7, weights_of=0), L(9, 9, 16, 8, 33, 72)], eps=1e-3),
        # one head per key/value head, odd sizes everywhere, window of one token (a large eps: a sublayer whose output
        # happens to be nearly zero for a token would otherwise be blown up by its output norm, rounding included)
        "odd": synth.layered_config(97, 75, [L(3, 3, 13, 7, 1, 51, scale=0.4), L(3, 3, 13, 7, 50, 51, coef=0.7, every=3), L(5, 1, 20, 9, 23, 33)], eps=2e-2),
        # many query heads on one key/value head, wide heads, a window longer than the prompts
        "wide": synth.layered_config(130, 192, [L(20, 2, 72, 136, 400, 96, coef=0.25, every=100), L(12, 1, 136, 72, 65, 320, weights_of=None)]),
        # a temperature that does nothing and one that does, value size equal to the key size
        "plain": synth.layered_config(64, 64, [L(2, 1, 32, 32, 16, 64, coef=0.0, every=1), L(2, 2, 32, 32, 17, 64, coef=1.0, every=1)], eps=1e-6),
    }


def build(synth, tmp_path, name, seed=0):
    cfg = variants(synth)[name]
    rng = np.random.default_rng(seed + sum(map(ord, name)))
    w = synth.layered_weights(rng, cfg)
    folder = tmp_path / f"{name}_{seed}"
    synth.write_layered(folder, cfg, w)
    return cfg, w, folder


def error(got, want):
    """Largest root-mean-square deviation of a row of logits (its mean taken off), in units of the logits' spread."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    d = got - want
    d -= d.mean(-1, keepdims=True)
    return float(np.sqrt((d * d).mean(-1)).max() / want.std())


TOL = {6: 0.02, 0: 2e-5}            # by dtype of the device model: bfloat16, float32


def reference(cfg, w, tokens):
    return lm_oracle.Model(cfg, w).forward(tokens)


def cut(n, sizes):
    """Splits range(n) into portions whose sizes are taken from `sizes` in turn."""
    at, i, out = 0, 0, []
    while at < n:
        k = min(sizes[i % len(sizes)], n - at)
        out.append((at, at + k))
        at += k
        i += 1
    return out
