"""Small layered models for the tests, and running them on the device and in the plain restatement."""
import numpy as np

import latent_oracle
import lenedra_oracle
import lm_oracle
import zevilorn_oracle


def variants(synth):
    """name -> configuration. Sizes are chosen so that no two of them coincide by accident."""
    L, A = synth.layered_layer, synth.latent_layer
    K, P, R = synth.kept_layer, synth.parallel_layer, synth.routed_mlp
    T, Q, G, S = synth.talking_layer, synth.queried_layer, synth.recurrent_layer, synth.sigmoid_mlp
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
        # latents: full and windowed layers, gates, frequency scaling, caches read by later layers with other head counts (one of
        # them two layers on), experts with 2 of 5, all and one chosen, a layer without feed-forward
        "latent": synth.latent_config(211, 144, [A(5, 24, 8, 40, 56, 200), A(3, 40, 24, 16, 72, (5, 2, 40, 0.8), 19, True, 3e4, (4.0, 64, 8.0, 1.0)),
                                                 A(7, 16, 8, 8, 56, None, kv_from=0), A(2, 24, 16, 24, 40, (3, 3, 33, 1.1), 70, True, 500.0),
                                                 A(4, 32, 8, 24, 56, (4, 1, 72, 2.0), kv_from=0, scale=0.3)], eps=1e-3),
        # odd sizes everywhere, a window of one token, every layer with a window, one pair of rotated dimensions
        "latent_odd": synth.latent_config(97, 75, [A(3, 13, 6, 7, 21, 51, 33), A(1, 5, 2, 9, 17, (7, 1, 17, 0.5), 1, True, 100.0),
                                                   A(5, 11, 6, 3, 21, 51, 50, kv_from=0), A(3, 3, 10, 21, 33, (2, 1, 45, 3.0), 23, True, 1e3, (1.0, 32, 4.0, 0.5))],
                                          eps=2e-2),
        # many heads, wide latents
        "latent_wide": synth.latent_config(130, 192, [A(20, 72, 64, 136, 300, 320, base=1e6), A(12, 104, 32, 72, 200, (40, 3, 48, 1.0), 90, True, 1e4, (8.0, 40, 16.0, 2.0))]),
        # sizes with tiles of their own, more than 64 (token, head) pairs per token
        "latent_full": synth.latent_config(64, 128, [A(4, 128, 64, 128, 512, 96, base=1e5), A(70, 8, 8, 8, 128, (9, 4, 24, 1.5), 40, True)]),
        # streams: every mechanism, key heads shared on both sides, value sizes of their own, a layer without feed-forward, windows and
        # chunks of different sizes, identity experts, one of them with all groups open
        "streams": synth.streams_config(211, 144, 3, [K(6, 3, 24, 19, 5, 200), P((6, 2, 24, 40, 37), (4, 2, 24, 32, 3), (12, 20), R(7, 3, 3, 5, 2, 40, 56)),
                                                       K(4, 1, 32, 70, 33, None), P((3, 3, 16, 8, 64), (5, 5, 40, 16, 5), (9, 33), R(4, 0, 2, 1, 1, 33, 17)),
                                                       K(5, 5, 16, 30, 1, R(6, 2, 5, 4, 4, 24, 72, 0.7))], eps=1e-3, scale=0.75),
        # odd sizes everywhere, a window of one token with more kept than it, a chunk of one, a convolution of one tap, one stream
        "streams_odd": synth.streams_config(97, 75, 1, [P((3, 1, 13, 7, 23), (3, 1, 11, 9, 2), (5, 3), 51, (-0.7, 0.4)), K(3, 3, 7, 1, 9, R(3, 4, 3, 7, 4, 17, 33, 2.5)),
                                                        P((5, 5, 9, 21, 1), (6, 3, 5, 3, 1), (1, 2), None), K(9, 3, 13, 50, 0, 33)], eps=2e-2, scale=0.7, cap=3.0),
        # wide heads, many heads, many streams, a window and a chunk longer than the prompts
        "streams_wide": synth.streams_config(130, 192, 6, [K(12, 4, 136, 400, 16, 96), P((20, 2, 72, 136, 500), (9, 3, 136, 200, 4), (24, 130), R(40, 8, 6, 12, 5, 48, 320, 1.0)),
                                                            K(3, 3, 40, 90, 2, R(5, 3, 3, 2, 1, 24, 33)), K(2, 1, 16, 25, 7, R(60, 0, 4, 6, 3, 17, 40))], cap=12.0),
        # sizes with tiles of their own; chunks and windows that end where blocks and tiles do
        "streams_full": synth.streams_config(64, 128, 4, [P((4, 2, 64, 64, 64), (2, 1, 128, 128, 4), (16, 16), R(9, 3, 4, 3, 2, 24, 24)), K(2, 1, 128, 64, 16, 96),
                                                          P((4, 4, 128, 128, 16), (4, 4, 64, 64, 4), (64, 64), 64)]),
        # sublayers side by side: every mixer, a loop over some of them, key heads shared, part of a head rotated, both ways to scale
        # frequencies and neither, a layer without feed-forward, groups and none
        "loops": synth.looped_config(211, 144, [T(6, 3, 24, 40, 37, 3, 4.0, S(8, 2, 40, (4, 2)), (16, 500.0), (3.0, 1.0, 4.0, 100)), Q(5, 24, 8, 40, 56, 40, S(6, 3, 33)),
                                                G((4, 2, 32, 24, 23), (8, 2000.0), 56, None, 2.5), T(4, 1, 16, 24, 70, 4, 2.5, S(9, 1, 24, (3, 1)), (16, 300.0)),
                                                G((3, 3, 24, 40, 90), (24, 900.0), 130, S(7, 7, 17))], (1, 4, 3), eps=1e-3),
        # odd sizes everywhere, one pair rotated, one tap and many, windows of one token, a loop from the first layer to the last
        "loops_odd": synth.looped_config(97, 75, [G((3, 1, 13, 7, 1), (2, 50.0), 37, S(5, 2, 51, (5, 2))), T(9, 3, 11, 5, 50, 1, 1.5, S(3, 1, 17), (6, 60.0), (2.0, 0.5, 3.0, 40)),
                                                  Q(3, 13, 6, 7, 21, 33, None, 100.0), T(1, 1, 7, 9, 1, 7, 3.0, None, (2, 10.0)), Q(1, 5, 2, 9, 3, 17, S(4, 2, 33, (2, 1)))], (0, 5, 2), eps=2e-2),
        # many heads, wide heads and latents, windows longer than the prompts, no loop
        "loops_wide": synth.looped_config(130, 192, [T(40, 8, 40, 72, 400, 4, 6.0, S(40, 5, 48, (8, 3)), (40, 1e4), (8.0, 1.0, 4.0, 64)), Q(20, 72, 64, 136, 200, 300, S(5, 2, 96)),
                                                     G((12, 4, 136, 200, 300), (64, 1e4), 320, S(12, 3, 40, (2, 2)), 4.0), T(100, 4, 8, 8, 65, 2, 2.0, None, (8, 100.0))]),
        # sizes with tiles of their own; windows that end where blocks and tiles do; a loop of one pass in front of a layer
        "loops_full": synth.looped_config(64, 128, [Q(4, 128, 64, 128, 64, 512, S(9, 4, 24, (3, 2))), G((4, 2, 64, 64, 64), (64, 1e4), 64, S(4, 2, 64, (4, 3))),
                                                    T(8, 4, 64, 128, 16, 3, 5.0, S(16, 2, 16, (2, 1)), (32, 1e3)), G((2, 1, 128, 128, 128), (32, 1e4), 128, None)], (1, 2, 1)),
        # windows in every layer, so that blocks are let go
        "loops_windows": synth.looped_config(90, 80, [T(4, 2, 24, 16, 33, 3, 3.0, S(4, 2, 24, (2, 1)), (12, 200.0)), G((2, 1, 16, 24, 70), (16, 500.0), 40, S(3, 2, 20))], (0, 1, 2), eps=1e-3),
        "plain": synth.layered_config(64, 64, [L(2, 1, 32, 32, 16, 64, coef=0.0, every=1), L(2, 2, 32, 32, 17, 64, coef=1.0, every=1)], eps=1e-6),
    }


def clear_groups(z, groups):
    """Whether the groups picked by the sum of their two best sigmoids lead by more than rounding, whatever the row's norm."""
    if not groups or groups["keep"] == groups["count"]:
        return True
    for scale in np.geomspace(0.05, 2.0, 20):
        two = np.sort(zevilorn_oracle.sigmoid(z * scale).reshape(groups["count"], -1), -1)[:, -2:].sum(-1)
        order = np.sort(two)[::-1]
        if order[groups["keep"] - 1] - order[groups["keep"]] < 0.02 * scale:
            return False
    return True


def steady_routes(synth, rng, cfg, w):
    """Makes the experts' choice independent of rounding: the routers read only the last columns of the residual, which
    hold well separated levels in an order of each token's own and which no sublayer adds to (identity experts and the
    mixing of streams only scale them)."""
    moe = [i for i, l in enumerate(cfg["layers"]) if (l["mlp"] or {}).get("kind") == "moe"]
    if not moe:
        return
    n = max(len(w[f"l{i}.mlp.router"]) for i in moe)
    level = (np.arange(n) - n / 2) * min(0.5, 4.0 / n)
    orders = {i: rng.permutation(n)[:len(w[f"l{i}.mlp.router"])] for i in moe}
    side = cfg["architecture"] == "Zevilorn"
    if side:
        level = level * 2
    rows, tries = [], 0
    while len(rows) < cfg["vocab"]:
        row, tries = rng.permutation(level), tries + 1
        assert tries < 200 * cfg["vocab"], "no order of levels separates the groups of every layer"
        if not side or all(clear_groups(row[o], cfg["layers"][i]["mlp"]["router"].get("groups")) for i, o in orders.items()):
            rows.append(row)
    w["embed"][:, -n:] = synth.bf16_round(np.stack(rows))[1]
    for name in w:
        if side:
            if name.endswith(".norm1"):
                w[name][-n:] = 1.0
            elif name.endswith((".o", ".o.b", ".down", ".out")):
                w[name][-n:] = 0.0
            continue
        if "streams" in cfg and name.endswith((".norm1", ".norm2", "mix.o.b")):
            w[name][-n:] = 0.0
        elif "streams" in cfg and name[0] == "l" and name.endswith((".o", ".down")):
            w[name][-n:] = 0.0
        elif name.endswith((".norm1", ".norm2")):
            w[name][-n:] = 0.0
            w[name] *= 0.5                             # rounding errors then grow little from layer to layer
    for i in moe:
        r = w[f"l{i}.mlp.router"]
        r[:] = 0.0
        r[np.arange(len(r)), cfg["width"] - n + orders[i]] = 1.0


def build(synth, tmp_path, name, seed=0):
    cfg = variants(synth)[name]
    rng = np.random.default_rng(seed + sum(map(ord, name)))
    w = synth.layered_weights(rng, cfg)
    steady_routes(synth, rng, cfg, w)
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


def model(cfg, w):
    """The plain restatement of a configuration's design."""
    return {"Rarolorn": lm_oracle, "Situlorn": latent_oracle, "Lenedra": lenedra_oracle, "Zevilorn": zevilorn_oracle}[cfg["architecture"]].Model(cfg, w)


def reference(cfg, w, tokens):
    return model(cfg, w).forward(tokens)


def cut(n, sizes):
    """Splits range(n) into portions whose sizes are taken from `sizes` in turn."""
    at, i, out = 0, 0, []
    while at < n:
        k = min(sizes[i % len(sizes)], n - at)
        out.append((at, at + k))
        at += k
        i += 1
    return out
