"""Talking heads over convolved and rotated projections, rotated windowed heads, attention over latents with sinks, the minimal gated
recurrence, gated joins and sigmoid routing: each kernel against the plain restatement (zevilorn_oracle.py). Projections are made
directly, so that single keys can be made to stand out just inside and just outside a window, at block borders and far away."""
import ctypes as C

import numpy as np
import pytest

import lm_util
import zevilorn_oracle as ze

pytestmark = pytest.mark.gpu
BS = 16
RNG = lambda s: np.random.default_rng(s)
pad = lambda n, to: (n + to - 1) // to * to
P = lambda t, k=0: t.data_ptr() + k


def up(a, dev, dtype=np.float32):
    import torch
    return torch.from_numpy(np.ascontiguousarray(a, dtype)).to(dev)


def sync():
    import torch
    torch.cuda.synchronize()


def tol(f32):
    return 2e-5 if f32 else 1.5e-2


class Heads:
    """Random projections of `lengths` tokens per sequence, a shuffled block table, device pools that hold nothing yet.
    talking: convolved, capped, mixed scores with a sink of one; otherwise plain windowed heads with a gate per head."""

    def __init__(self, pkg, dev, m, lengths, f32, seed=0, talking=True, room=None, identity=False):
        import torch
        self.pkg, self.dev, self.m, self.f32, self.talking, self.room = pkg, dev, m, f32, talking, room
        H, G, D, V, T = (m[k] for k in ("heads", "kv_heads", "dim", "vdim", "conv"))
        r = RNG(seed)
        self.qw, self.kw, self.vw = H * D, G * D, G * V
        self.cols = self.qw + self.kw + self.vw + (0 if talking else H)
        self.rows = [r.standard_normal((n, self.cols)).astype(np.float32) for n in lengths]
        ch = self.qw + self.kw + self.vw
        self.taps = (r.standard_normal((ch, T)) / max(T, 1) ** 0.5).astype(np.float32) if talking else None
        self.talk = (0.6 * np.eye(H) + r.standard_normal((H, H)) / H ** 0.5).astype(np.float32)
        if identity:
            self.taps[:] = np.eye(T)[-1]
            self.talk = np.eye(H, dtype=np.float32)
        self.freq = ze.frequencies(m["rot"]).astype(np.float32)
        per = max(pad(n, BS) // BS for n in lengths)
        ids = r.permutation(per * len(lengths) + 3)
        self.table = np.zeros((len(lengths), per + 1), np.int32)
        for s in range(len(lengths)):
            self.table[s, :per] = ids[s * per:(s + 1) * per]
        t = torch.float32 if f32 else torch.float16
        nan = lambda *shape, dtype=torch.float32: torch.full(shape, float("nan"), dtype=dtype, device=dev)         # nothing but what was written may be read
        self.kp, self.vp = (nan(len(ids) * BS, G, pad(d, 16), dtype=t) for d in (D, V))
        self.ring = nan(len(lengths), max(T, 1), ch)
        self.keep = [up(self.freq, dev), up(self.table, dev, np.int32), up(self.taps.T if talking else [0], dev), up(self.talk, dev)]
        a = self.a = pkg.Attn(H, G, D, V, pad(D, 16), pad(V, 16), m["scale"], m["mask"]["size"], None, int(talking), None, None, 0, 0, 0, -1 if talking else ch,
                              pkg.DT_F32 if f32 else pkg.DT_F16, P(self.kp), P(self.vp), BS, P(self.keep[1]), self.table.shape[1])
        a.freq, a.rot_dims = P(self.keep[0]), m["rot"]["dims"]
        if talking:
            a.taps, a.conv, a.ring, a.cap, a.talk = T, P(self.keep[2]), P(self.ring), m["softcap"], P(self.keep[3])

    def want(self, s):
        m, x = self.m, self.rows[s].astype(np.float64)
        n, H, G, D = len(x), m["heads"], m["kv_heads"], m["dim"]
        pos, gate = np.arange(n), 1.0
        if self.talking:
            x, _ = ze.causal_conv(x, self.taps.astype(np.float64), np.zeros((m["conv"] - 1, x.shape[1])))
        else:
            gate = ze.sigmoid(x[:, -H:])[:, :, None]
            x = x[:, :-H]
        f = self.freq.astype(np.float64)
        q, k = (ze.rotate_neighbours(p.reshape(n, -1, D), pos, f) for p in (x[:, :self.qw], x[:, self.qw:self.qw + self.kw]))
        z = ze.scores(q, k, m["scale"])
        if self.talking:
            z = ze.mix_heads(ze.soft_cap(z, m["softcap"]), self.talk.astype(np.float64))
        p = ze.weights_over(z, ze.window(pos, pos, m["mask"]["size"]), np.zeros(H) if self.talking else None)
        return (ze.weighted_values(p, x[:, self.qw + self.kw:].reshape(n, G, -1)) * gate).reshape(n, -1)

    def talking_step(self, d, ld, dp, ds, dt, tiles, runs, one, n, keys, out, ow):
        import torch
        pkg, L, a, m = self.pkg, self.pkg.lib, self.a, self.m
        H, dl = m["heads"], pad(m["dim"], 16)
        q = torch.full((n, H, dl), float("nan"), dtype=torch.float32 if self.f32 else torch.float16, device=self.dev)
        pkg.check(L.cmlb200_rotate_append(a, P(d), ld, P(dp), P(ds), 0, n, one, P(q), None))
        if len(runs):
            dr = up(runs, self.dev, np.int32)
            pkg.check(L.cmlb200_ring_rows(a, P(d), ld, P(dr), len(runs), None))
        sl = pad(min(m["mask"]["size"] + 79, keys + 15), 64)
        at_once = self.room or max(1, n, tiles)
        buf = torch.full((at_once, H, 1 if self.f32 else 64, sl), float("nan"), device=self.dev)
        b = pkg.Attn.from_buffer_copy(a)
        b.scores, b.scores_ld = P(buf), sl
        if self.f32:
            for r in range(0, n, at_once):
                k = min(at_once, n - r)
                pkg.check(L.cmlb200_talk_scores_rows(a, P(q, 4 * r * H * dl), P(dp, 4 * r), P(ds, 4 * r), k, keys, P(buf), sl, None))
                pkg.check(L.cmlb200_attention_rows_f32(b, P(d, 4 * r * ld), ld, P(dp, 4 * r), P(ds, 4 * r), k, P(out, 4 * r * ow), ow, None))
            return
        for t in range(0, tiles, at_once):
            k = min(at_once, tiles - t)
            pkg.check(L.cmlb200_talk_scores_tiles(a, P(q), P(dt, 16 * t), k, keys, P(buf), sl, None))
            pkg.check(L.cmlb200_attention_tiles(b, P(d), ld, P(dt, 16 * t), k, P(out), ow, None))
        if one:
            pkg.check(L.cmlb200_talk_scores_rows(a, P(q), P(dp), P(ds), one, keys, P(buf), sl, None))
            pkg.check(L.cmlb200_attention_one(b, P(d), ld, P(dp), P(ds), one, keys, P(out), ow, None))

    def windowed_step(self, d, ld, dp, ds, dt, tiles, one, n, keys, out, ow):
        pkg, L, a = self.pkg, self.pkg.lib, self.a
        if self.f32:
            pkg.check(L.cmlb200_rotate_append(a, P(d), ld, P(dp), P(ds), 0, n, 0, None, None))
            pkg.check(L.cmlb200_attention_rows_f32(a, P(d), ld, P(dp), P(ds), n, P(out), ow, None))
            return
        if n > one:
            pkg.check(L.cmlb200_rotate_append(a, P(d), ld, P(dp), P(ds), one, n - one, one, None, None))
            pkg.check(L.cmlb200_attention_tiles(a, P(d), ld, P(dt), tiles, P(out), ow, None))
        if one:
            pkg.check(L.cmlb200_attention_one(a, P(d), ld, P(dp), P(ds), one, keys, P(out), ow, None))

    def run(self, steps):
        """steps: lists of (sequence, first, end); single tokens come first among a step's rows."""
        import torch
        ow = self.m["heads"] * self.m["vdim"]
        got = [np.full((len(x), ow), np.nan) for x in self.rows]
        for step in steps:
            step = sorted(step, key=lambda p: p[2] - p[1] > 1)
            one = sum(e - b == 1 for _, b, e in step)
            x = np.concatenate([self.rows[s][b:e] for s, b, e in step])
            n, ld = len(x), x.shape[1] + (3 if self.m["heads"] % 2 else 4)
            buf = np.zeros((n, ld), np.float32)
            buf[:, :x.shape[1]] = x
            tiles, runs, at = [], [], one
            for s, b, e in step[one:]:
                runs.append([at, e - b, s, b])
                tiles += [[at + k, min(64, e - b - k), s, b + k] for k in range(0, e - b, 64)]
                at += e - b
            d, dp = up(buf, self.dev), up(np.concatenate([np.arange(b, e) for _, b, e in step]), self.dev, np.int32)
            ds, dt = up(np.concatenate([np.full(e - b, s) for s, b, e in step]), self.dev, np.int32), up(tiles or [[0] * 4], self.dev, np.int32)
            out = torch.zeros((n, ow + 5), device=self.dev, dtype=torch.float32 if self.f32 else torch.bfloat16)
            keys = max(e for _, _, e in step)
            if self.talking:
                self.talking_step(d, ld, dp, ds, dt, len(tiles), runs, one, n, keys, out, ow + 5)
            else:
                self.windowed_step(d, ld, dp, ds, dt, len(tiles), one, n, keys, out, ow + 5)
            sync()
            o, at = out.float().cpu().numpy(), 0
            assert (o[:, ow:] == 0).all()
            for s, b, e in step:
                got[s][b:e] = o[at:at + e - b, :ow]
                at += e - b
        return got


def heads(H, G, D, V, window, taps, cap, rot, scale=None):
    return {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale or D ** -0.5, "mask": {"size": window}, "conv": taps, "softcap": cap, "rot": {"dims": rot, "base": 100.0}}


def schedules(lengths, seed=3):
    """Whole prompts, single tokens, portions of two, and a random mixture."""
    out = [[[(s, 0, n) for s, n in enumerate(lengths)]], [[(s, t, t + 1) for s, n in enumerate(lengths) if t < n] for t in range(max(lengths))],
           [[(s, t, min(t + 2, n)) for s, n in enumerate(lengths) if t < n] for t in range(0, max(lengths), 2)]]
    r, at, mix = RNG(seed), [0] * len(lengths), []
    while any(a < n for a, n in zip(at, lengths)):
        step = []
        for s, n in enumerate(lengths):
            k = min(int(r.choice([0, 1, 1, 2, 3, 5, 16, 33, 64, 70, 90])), n - at[s])
            if k:
                step.append((s, at[s], at[s] + k))
                at[s] += k
        if step:
            mix.append(step)
    return out + [mix]


TALKING = [(4, 2, 32, 24, 23, 3, 3.0, 16), (3, 3, 13, 7, 1, 4, 1.5, 6), (20, 2, 72, 136, 100, 1, 5.0, 72), (8, 1, 64, 64, 64, 2, 4.0, 32), (2, 2, 128, 128, 65, 3, 6.0, 2),
           (6, 3, 200, 17, 40, 5, 2.0, 100), (1, 1, 256, 40, 17, 9, 2.0, 30), (64, 8, 16, 24, 70, 4, 3.0, 8), (110, 5, 8, 9, 33, 3, 2.0, 8), (5, 5, 16, 256, 1000, 3, 8.0, 16)]
WINDOWED = [(4, 2, 32, 24, 23, 0, 0, 16), (3, 3, 13, 7, 1, 0, 0, 6), (20, 2, 72, 136, 100, 0, 0, 72), (8, 1, 64, 64, 64, 0, 0, 32), (2, 2, 128, 128, 65, 0, 0, 2), (6, 3, 200, 256, 40, 0, 0, 100),
            (5, 5, 16, 80, 1000, 0, 0, 16)]


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("shape", TALKING + WINDOWED)
def test_attention_in_every_schedule(pkg, torch_dev, shape, f32):
    lengths = [130, 1, 65, 17]
    L = Heads(pkg, torch_dev, heads(*shape), lengths, f32, talking=shape[5] > 0)
    want = [L.want(s) for s in range(len(lengths))]
    for steps in schedules(lengths):
        for w, g in zip(want, L.run(steps)):
            assert np.abs(w - g).max() < tol(f32) * max(1, np.abs(w).max())


@pytest.mark.parametrize("f32", [False, True])
def test_scores_pass_a_few_rows_at_a_time(pkg, torch_dev, f32):
    L = Heads(pkg, torch_dev, heads(4, 2, 32, 24, 50, 3, 3.0, 16), [200, 70], f32, room=2)
    want = [L.want(s) for s in range(2)]
    for w, g in zip(want, L.run([[(0, 0, 199), (1, 0, 70)], [(0, 199, 200)]])):
        assert np.abs(w - g).max() < tol(f32) * 2


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("change", ["cap", "talk", "taps", "rotation"])
def test_every_mechanism_alone_shows(pkg, torch_dev, change, f32):
    """One of them neutral, the others as they are; and the neutral one is far from the full mechanism."""
    m = heads(6, 3, 32, 24, 40, 3, 1.5, 16)
    full = Heads(pkg, torch_dev, m, [90], f32)
    L = Heads(pkg, torch_dev, m, [90], f32)
    if change == "cap":
        L.m = dict(m, softcap=1e6)
        L.a.cap = 0.0
    elif change == "talk":
        L.talk, L.a.talk = np.eye(6, dtype=np.float32), None
    elif change == "taps":
        L.taps[:, :-1] = 0
        L.keep[2] = up(L.taps.T, torch_dev)
        L.a.conv = P(L.keep[2])
    else:
        L.freq = np.zeros_like(L.freq)
        L.keep[0] = up(L.freq, torch_dev)
        L.a.freq = P(L.keep[0])
    want = L.want(0)
    assert np.abs(want - full.want(0)).max() > 0.1
    for steps in schedules([90]):
        assert np.abs(want - L.run(steps)[0]).max() < tol(f32) * 2


def stand_out(L, pairs):
    """For each (query, key) position of sequence 0 every head's query points along the key in the entries that do not turn, strongly
    enough that the key takes nearly all the weight where it is seen."""
    m, x, r = L.m, L.rows[0], RNG(9)
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    for q, k in pairs:
        key = r.choice([-1.0, 1.0], (G, D))
        x[k, L.qw:L.qw + L.kw] = key.ravel()
        x[q, :L.qw] = np.repeat(key, H // G, axis=0).ravel()


def edges(L, f32, n, pairs, move):
    stand_out(L, pairs)
    want = L.want(0)
    for steps in ([[(0, 0, n)]], [[(0, t, min(t + 57, n))] for t in range(0, n, 57)],
                  [[(0, 0, 100)], [(0, 100, 102)], [(0, 102, 173)]] + [[(0, t, t + 1)] for t in range(173, n)], [[(0, 0, 2)]] + [[(0, t, t + 1)] for t in range(2, n)]):
        assert np.abs(want - L.run(steps)[0]).max() < tol(f32) * 3
    move()
    assert (np.abs(L.want(0) - want)[[q for q, _ in pairs]].max(1) > 6 * tol(f32)).all()


def disjoint(pairs):
    out, used = [], set()
    for q, k in pairs:
        if 0 <= k < q and not {q, k} & used:
            out.append((q, k))
            used |= {q, k}
    return out


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("talking", [True, False])
@pytest.mark.parametrize("size", [16, 17, 31, 33, 64, 80, 129])
def test_window_edges(pkg, torch_dev, size, talking, f32):
    """Distance size - 1 is seen, distance size is not; queries sit around block and tile borders."""
    n = 330
    for off, step in ((size - 1, -1), (size, 1)):
        qs = [q for q in (size + 9, size + 10, 63 + size, 64 + size, 160, 175, 192, 255, 256, 329) if q - off >= 0]
        L = Heads(pkg, torch_dev, heads(8, 2, 32, 24, size, 3 if talking else 0, 60.0, 8, 0.7), [n], f32, talking=talking, identity=talking)
        edges(L, f32, n, disjoint([(q, q - off) for q in qs]), lambda: L.m["mask"].update(size=size + step))


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("talking", [True, False])
def test_far_key_among_hundreds(pkg, torch_dev, talking, f32):
    n = 900
    pairs = [(q, k) for q, k in ((899, 0), (898, 15), (897, 16), (896, 31), (895, 32), (894, 63), (893, 64), (850, 127), (833, 128), (770, 511), (769, 300))]
    L = Heads(pkg, torch_dev, heads(4, 2, 32, 24, 1000, 2 if talking else 0, 80.0, 8, 0.8), [n], f32, talking=talking, identity=talking)
    stand_out(L, pairs)
    want = L.want(0)
    for steps in ([[(0, 0, n)]], [[(0, 0, 740)], [(0, 740, 800)], [(0, 800, n)]], [[(0, 0, 760)]] + [[(0, t, t + 1)] for t in range(760, n)]):
        assert np.abs(want - L.run(steps)[0]).max() < tol(f32) * 3
    for _, k in pairs:
        L.rows[0][k, L.qw:L.qw + L.kw] *= -1
    assert (np.abs(L.want(0) - want)[[q for q, _ in pairs]].max(1) > 20 * tol(f32)).all()


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("taps", [1, 2, 3, 4, 7])
def test_every_tap_across_every_cut(pkg, torch_dev, taps, f32):
    """A spike in one projection reaches exactly the next taps - 1 tokens, in whole prompts, portions of two and three, and decoding."""
    n = 70
    for spike in (0, 15, 16, 40, 63):
        L = Heads(pkg, torch_dev, heads(2, 1, 16, 16, 1, taps, 5.0, 4), [n], f32)
        L.rows[0][:] *= 0.01
        L.rows[0][spike, L.qw + L.kw:] = 30.0
        want = L.want(0)                               # a window of one: a token's own value and the sink
        hit = np.abs(want).max(1) > 0.1
        assert hit[spike:spike + taps].any() and not hit[:spike].any() and not hit[spike + taps:].any()
        for steps in ([[(0, 0, n)]], [[(0, t, min(t + 2, n))] for t in range(0, n, 2)], [[(0, t, min(t + 3, n))] for t in range(0, n, 3)], [[(0, t, t + 1)] for t in range(n)]):
            assert np.abs(want - L.run(steps)[0]).max() < tol(f32) * 30


def test_long_decode_splits_keys_over_a_cluster(pkg, torch_dev):
    n = 3000
    for talking, m in ((True, heads(8, 2, 64, 64, 2500, 3, 4.0, 32)), (False, heads(4, 4, 64, 48, 2990, 0, 0, 64))):
        L = Heads(pkg, torch_dev, m, [n], False, talking=talking)
        got = L.run([[(0, 0, n - 20)]] + [[(0, t, t + 1)] for t in range(n - 20, n)])[0]
        assert np.abs(L.want(0) - got)[n - 60:].max() < tol(False)


def test_refusals(pkg, torch_dev):
    lib = pkg.lib
    L = Heads(pkg, torch_dev, heads(4, 2, 32, 24, 50, 3, 3.0, 16), [20], False)
    d, i = up(np.zeros((4, 400)), torch_dev), up(np.zeros(16), torch_dev, np.int32)
    assert lib.cmlb200_rotate_append(L.a, P(d), 400, P(i), P(i), 0, 1, 1, None, None) != 0          # convolved queries need a place
    assert lib.cmlb200_rotate_append(L.a, P(d), 10, P(i), P(i), 0, 1, 1, P(d), None) != 0
    assert lib.cmlb200_talk_scores_tiles(L.a, P(d), P(i), 1, 500, P(d), 64, None) != 0               # the stride does not hold a window and a tile
    assert lib.cmlb200_talk_scores_rows(L.a, P(d), P(i), P(i), 1, 500, P(d), 48, None) != 0
    bad = pkg.Attn.from_buffer_copy(L.a)
    bad.rot_dims = 34
    assert lib.cmlb200_rotate_append(bad, P(d), 400, P(i), P(i), 0, 1, 1, P(d), None) != 0


# ---- attention over latents with sinks and a gate per head -----------------------------------------------------
@pytest.mark.parametrize("form", [1, 2])
@pytest.mark.parametrize("sink", [-8.0, 0.0, 4.0, 40.0])
def test_latents_with_sinks_in_either_form(pkg, synth, tmp_path, torch_dev, form, sink):
    """Single tokens, short portions and expanded ones agree about sinks that take nothing, a share, most, or all but nothing of the weight."""
    cfg = synth.looped_config(70, 96, [synth.queried_layer(5, 24, 8, 40, 48, 72, None), synth.queried_layer(3, 16, 4, 24, 20, 130, None)], eps=1e-3)
    w = synth.layered_weights(RNG(4), cfg)
    for i in (0, 1):
        w[f"l{i}.mix.sink"] = synth.bf16_round((sink + RNG(5).standard_normal(w[f"l{i}.mix.sink"].shape)).astype(np.float32))[1]
    synth.write_layered(tmp_path / "m", cfg, w)
    t = RNG(6).integers(0, 70, 300)
    want = lm_util.reference(cfg, w, t)
    without = dict(w, **{f"l{i}.mix.sink": np.full_like(w[f"l{i}.mix.sink"], -1e9) for i in (0, 1)})
    assert (lm_util.error(lm_util.reference(cfg, without, t), want) > 0.1) == (sink >= 0)
    pkg.check(pkg.lib.cmlb200_set_attention_latent_form(form))
    try:
        m = pkg.LanguageModel(tmp_path / "m", 6, max_tokens=320, max_sequences=1)
        for sizes in ([300], [33], [100, 64, 2, 1, 1], [200] + [1] * 100):
            s = m.open()
            got = np.concatenate([m.step([(s, t[a:b], None)])[0] for a, b in lm_util.cut(300, sizes)])
            m.end(s)
            assert lm_util.error(got, want) < lm_util.TOL[6]
        m.close()
    finally:
        pkg.lib.cmlb200_set_attention_latent_form(0)


# ---- minimal gated recurrence ------------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("width", [1, 33, 300])
def test_recurrence_in_every_schedule(pkg, torch_dev, width, f32):
    """States of empty slots hold anything. Gates reach from nearly closed to nearly open; what one token wrote long ago stays."""
    import torch
    lengths, col, r = [200, 1, 65, 33], 3, RNG(width)
    rows = [np.concatenate([4 * r.standard_normal((n, width)) - 2, r.standard_normal((n, 2 * width))], 1).astype(np.float32) for n in lengths]
    rows[0][:, 0] = -20.0                              # a gate that stays shut behind the first token
    rows[0][0, 0] = 20.0
    want = []
    for x in rows:
        z, u, g = (p.astype(np.float64) for p in np.split(x, 3, 1))
        want.append(ze.gated_scan(ze.sigmoid(z), ze.candidate(u), np.zeros(width)) * ze.silu(g))
    for steps in schedules(lengths):
        state = torch.full((4, width), float("nan"), device=torch_dev)
        a = pkg.Gru(width, col, P(state))
        for step in steps:
            step = sorted(step, key=lambda p: p[2] - p[1] > 1)
            one = sum(e - b == 1 for _, b, e in step)
            d = up(np.pad(np.concatenate([rows[s][b:e] for s, b, e in step]), ((0, 0), (col, 2))), torch_dev)
            runs, at = [], one
            for s, b, e in step[one:]:
                runs.append([at, e - b, s, b])
                at += e - b
            out = torch.zeros(len(d), width + 1, device=torch_dev, dtype=torch.float32 if f32 else torch.bfloat16)
            dp, ds = up([b for _, b, _ in step], torch_dev, np.int32), up([s for s, _, _ in step], torch_dev, np.int32)
            dtype = pkg.DT_F32 if f32 else pkg.DT_BF16
            if runs:
                dr = up(runs, torch_dev, np.int32)
                pkg.check(pkg.lib.cmlb200_gru_rows(a, P(d), d.shape[1], P(dr), len(runs), P(out), dtype, width + 1, None))
            if one:
                sync()
                pkg.check(pkg.lib.cmlb200_gru_one(a, P(d), d.shape[1], P(dp), P(ds), one, P(out), dtype, width + 1, None))
            sync()
            o, at = out.float().cpu().numpy(), 0
            assert (o[:, width] == 0).all()
            for s, b, e in step:
                w = want[s][b:e]
                assert np.abs(o[at:at + e - b, :width] - w).max() < (1e-5 if f32 else 1e-2) * max(1, np.abs(w).max())
                at += e - b


# ---- joins, norms, activations -----------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("rows,width", [(1, 64), (5, 75), (40, 1024), (700, 96), (3, 5000)])
@pytest.mark.parametrize("two,ff,again,norm", [(False, 0, False, True), (True, 1, False, True), (False, 1, True, True), (True, 3, True, True), (True, 0, False, False), (False, 2, True, False)])
def test_gated_join(pkg, torch_dev, rows, width, two, ff, again, norm, f32):
    import torch
    r, dev, eps, vocab = RNG(width + rows), torch_dev, 1e-2, 31
    g = lambda *s: r.standard_normal(s).astype(np.float32)
    x, a, b, f, gates, wa, wb, wn, table, tok = (g(rows, width), g(rows, width), 3 * g(rows, width), g(rows * max(ff, 1) + 2, width), g(rows, 2 * width), g(width), g(width), g(width),
                                                 lm_util_round(g(vocab, width)), r.integers(0, vocab, rows))
    pos, wt = r.permutation(rows * max(ff, 1) + 2)[:rows * max(ff, 1)], r.random(rows * max(ff, 1)).astype(np.float32)
    d64 = lambda v: v.astype(np.float64)
    m = ze.normed_half_sum(d64(a), d64(b), d64(wa), d64(wb), eps) if two else d64(a)
    want = d64(x) + ze.sigmoid(d64(gates[:, :width])) * m
    if ff:
        y = d64(f[:rows]) if ff == 1 else (d64(wt)[:, None] * d64(f[pos])).reshape(rows, ff, width).sum(1)
        want = want + ze.sigmoid(d64(gates[:, width:])) * y
    if again:
        want = want + d64(table[tok])
    keep = {k: up(v, dev) for k, v in dict(x=x, a=a, b=b, f=f, gates=gates, wa=wa, wb=wb, wn=wn, table=table, wt=wt).items()}
    t16, ti, tp = keep["table"].bfloat16(), up(tok, dev, np.int32), up(pos, dev, np.int32)
    moe = pkg.Moe(8, ff, pos=P(tp), weight=P(keep["wt"]))
    j = pkg.GatedJoin(P(keep["a"]), P(keep["b"]) if two else None, width, P(keep["wa"]) if two else None, P(keep["wb"]) if two else None, P(keep["f"]) if ff else None, width,
                      C.pointer(moe) if ff > 1 else None, P(keep["gates"]), P(keep["gates"], 4 * width), 2 * width,
                      (P(keep["table"]) if f32 else P(t16)) if again else None, pkg.DT_F32 if f32 else pkg.DT_BF16, vocab, P(ti) if again else None)
    out = torch.zeros(rows, width + 3, device=dev, dtype=torch.float32 if f32 else torch.bfloat16)
    pkg.check(pkg.lib.cmlb200_gated_join_rows(j, P(keep["x"]), P(keep["wn"]) if norm else None, eps, rows, width, P(out), pkg.DT_F32 if f32 else pkg.DT_BF16, width + 3, None))
    sync()
    assert np.abs(keep["x"].cpu().numpy() - want).max() < 1e-5 * max(1, np.abs(want).max())
    n = ze.rms_norm(want, d64(wn), eps) if norm else np.zeros_like(want)
    o = out.float().cpu().numpy()
    assert np.abs(o[:, :width] - n).max() < (2e-5 if f32 else 2e-2) * max(1, np.abs(n).max()) and (o[:, width:] == 0).all()


def lm_util_round(a):
    """Nearest bf16 values."""
    import torch
    return torch.from_numpy(a).bfloat16().float().numpy()


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("n,col", [(1, 0), (40, 7), (1536, 64)])
def test_norm_of_columns(pkg, torch_dev, n, col, f32):
    import torch
    r = RNG(n)
    x, w = r.standard_normal((9, col + n + 5)).astype(np.float32), r.standard_normal(n).astype(np.float32)
    d, dw, out = up(x, torch_dev), up(w, torch_dev), torch.zeros(9, n + 2, device=torch_dev, dtype=torch.float32 if f32 else torch.bfloat16)
    pkg.check(pkg.lib.cmlb200_norm_columns(P(d), x.shape[1], col, n, P(dw), 1e-2, 9, P(out), pkg.DT_F32 if f32 else pkg.DT_BF16, n + 2, None))
    sync()
    want = ze.rms_norm(x[:, col:col + n].astype(np.float64), w, 1e-2)
    o = out.float().cpu().numpy()
    assert np.abs(o[:, :n] - want).max() < (1e-5 if f32 else 2e-2) * max(1, np.abs(want).max()) and (o[:, n:] == 0).all()


ACTS = {0: ze.silu, 1: lambda z: 0.5 * z * (1 + np.tanh(np.sqrt(2 / np.pi) * (z + 0.044715 * z ** 3))), 3: ze.gelu_erf}


@pytest.mark.parametrize("act", list(ACTS))
def test_activation_of_rows(pkg, torch_dev, act):
    import torch
    z = np.linspace(-12, 12, 1003).astype(np.float32).reshape(1, -1)
    d, f = up(z, torch_dev), torch.zeros(1, 1003, device=torch_dev)
    pkg.check(pkg.lib.cmlb200_act_rows_f32(P(d), 1003, 1, 1003, act, P(f), 1003, None))
    sync()
    assert np.abs(f.cpu().numpy() - ACTS[act](z.astype(np.float64))).max() < 3e-6
    assert pkg.lib.cmlb200_act_rows_f32(P(d), 1003, 1, 1003, 2, P(f), 1003, None) != 0               # needs a gate


# ---- routing and experts without a gate ----------------------------------------------------------------------------
def plan(pkg, dev, E, top, rows, align):
    import torch
    n = pkg.lib.cmlb200_moe_positions(rows, top, E, align)
    i = lambda k: torch.zeros(k, device=dev, dtype=torch.int32)
    t = {"ids": i(rows * top), "weight": torch.zeros(rows * top, device=dev), "pos": i(rows * top), "src": i(n), "expert": i(n), "start": i(E), "count": i(E), "active": i(E), "num_active": i(1),
         "tiles": i(4 * (n // 128 + E + 1)), "num_tiles": i(1)}
    return t, pkg.Moe(E, top, **{k: P(v) for k, v in t.items()}), n


@pytest.mark.parametrize("rows", [1, 7, 32, 33, 300])
@pytest.mark.parametrize("E,top,groups", [(16, 2, (4, 2)), (9, 3, (3, 2)), (12, 5, (12, 6)), (64, 6, (8, 4)), (40, 40, None), (7, 1, None), (6, 6, (2, 2))])
def test_routing_by_sigmoids(pkg, torch_dev, rows, E, top, groups):
    r = RNG(rows * E + top)
    z = r.standard_normal((rows, E)).astype(np.float32) * 2
    router = {"top": top, "experts": E}
    if groups:
        router["groups"] = dict(zip(("count", "keep"), groups))
    ids, p = ze.route(z.astype(np.float64), {"router": np.eye(E)}, router)
    t, m, _ = plan(pkg, torch_dev, E, top, rows, 1)
    m.sigmoid, m.group_best = 1, 2
    if groups:
        m.groups, m.keep = groups
    d = up(np.pad(z, ((0, 0), (0, 3))), torch_dev)
    pkg.check(pkg.lib.cmlb200_moe_route(m, P(d), E + 3, rows, 1, None))
    sync()
    assert (t["ids"].cpu().numpy().reshape(rows, top) == ids).all()
    assert np.abs(t["weight"].cpu().numpy().reshape(rows, top) - p).max() < 1e-6


@pytest.mark.parametrize("act", list(ACTS))
@pytest.mark.parametrize("rows,E,top,W,ff", [(1, 5, 2, 96, 40), (20, 9, 3, 64, 17), (32, 3, 1, 200, 64), (150, 6, 2, 128, 33), (400, 2, 2, 72, 130)])
def test_experts_without_a_gate(pkg, torch_dev, rows, E, top, W, ff, act):
    import torch
    r, dev, lib = RNG(rows + ff), torch_dev, pkg.lib
    x, u = lm_util_round(r.standard_normal((rows, W)).astype(np.float32)), lm_util_round((r.standard_normal((E, ff, W)) / W ** 0.5).astype(np.float32))
    align = 1 if rows <= 32 else 128
    t, m, n = plan(pkg, dev, E, top, rows, align)
    m.sigmoid = 1
    z = up(r.standard_normal((rows, E)), dev)
    pkg.check(lib.cmlb200_moe_route(m, P(z), E, rows, align, None))
    fp, ld = pad(ff, 16), pad(W, 64)
    w = np.zeros((E, fp, ld), np.float32)
    w[:, :ff, :W] = u
    dw, dx = up(w, dev).bfloat16(), up(np.pad(x, ((0, 0), (0, ld - W))), dev).bfloat16()
    D = pkg.Dense(pkg.DT_BF16, E * fp, W, ld, P(dw), None, 0.0)
    f = torch.zeros(n, pad(ff, 64), device=dev, dtype=torch.bfloat16)
    if rows <= 32:
        pkg.check(lib.cmlb200_moe_gemv_act(m, D, P(dx), ld, 1, rows, ff, act, P(f), f.shape[1], None))
    else:
        xp = torch.zeros(n, ld, device=dev, dtype=torch.bfloat16)
        pkg.check(lib.cmlb200_moe_gather(m, P(dx), ld, rows, W, P(xp), ld, None))
        pkg.check(lib.cmlb200_moe_gemm_act(m, D, P(xp), ld, rows, ff, act, P(f), f.shape[1], None))
    sync()
    ids, pos, o = t["ids"].cpu().numpy(), t["pos"].cpu().numpy(), f.float().cpu().numpy()
    for k in range(rows * top):
        want = ACTS[act](u[ids[k]].astype(np.float64) @ x[k // top].astype(np.float64))
        assert np.abs(o[pos[k], :ff] - want).max() < 1e-2 * max(1, np.abs(want).max())
