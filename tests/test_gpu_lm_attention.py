"""Attention over paged caches, each kernel against the plain restatement. The projections of a test are
made directly, so that single keys can be made to stand out just inside and just outside a window, at block
borders and far away."""
import numpy as np
import pytest

import lm_oracle as lo

pytestmark = pytest.mark.gpu
BS = 16


class Layer:
    """Random projections of `lengths` tokens per sequence for a mixer, a shuffled block table and device pools."""

    def __init__(self, pkg, dev, mixer, lengths, f32, seed=0, sink=True, bias=True, gate=True, norm=True):
        import torch
        self.pkg, self.dev, self.m, self.f32 = pkg, dev, mixer, f32
        H, G, D, V = (mixer[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        r = np.random.default_rng(seed)
        self.flags = dict(sink=sink, bias=bias, gate=gate, norm=norm)
        self.qw, self.kw, self.vw = H * D, G * D, G * V
        self.rows = [r.standard_normal((n, self.qw + self.kw + self.vw + H)).astype(np.float32) for n in lengths]
        self.qn, self.kn = ((1 + 0.3 * r.standard_normal(n)).astype(np.float32) for n in (self.qw, self.kw))
        self.eps = 1e-3
        up = lambda a: torch.from_numpy(np.ascontiguousarray(a)).to(dev)
        per = max((n + BS - 1) // BS for n in lengths)
        ids = r.permutation(per * len(lengths) + 3)
        self.table = np.zeros((len(lengths), per + 1), np.int32)
        for s in range(len(lengths)):
            self.table[s, :per] = ids[s * per:(s + 1) * per]
        pad = lambda n: (n + 15) // 16 * 16
        dt = torch.float32 if f32 else torch.float16
        nan = float("nan")                            # nothing but written slots may be read
        self.kp = torch.full((len(ids) * BS, G, pad(D)), nan, dtype=dt, device=dev)
        self.vp = torch.full((len(ids) * BS, G, pad(V)), nan, dtype=dt, device=dev)
        self.keep = [up(self.qn), up(self.kn), up(lo.alibi_slopes(H).astype(np.float32)), up(self.table)]
        t = mixer.get("q_temp") or {"coef": 0, "every": 0}
        self.a = pkg.Attn(H, G, D, V, pad(D), pad(V), mixer["scale"], mixer["mask"]["size"], self.keep[2].data_ptr() if bias else None, int(sink),
                          self.keep[0].data_ptr() if norm else None, self.keep[1].data_ptr() if norm else None, self.eps, t["coef"], t["every"],
                          self.qw + self.kw + self.vw if gate else -1, pkg.DT_F32 if f32 else pkg.DT_F16, self.kp.data_ptr(), self.vp.data_ptr(), BS,
                          self.keep[3].data_ptr(), self.table.shape[1])

    def want(self, s):
        """[n, H * vdim] of the whole sequence, from the restatement."""
        m, x = self.m, self.rows[s].astype(np.float64)
        n, H, G = len(x), m["heads"], m["kv_heads"]
        q, k, v = x[:, :self.qw], x[:, self.qw:self.qw + self.kw], x[:, self.qw + self.kw:self.qw + self.kw + self.vw]
        if self.flags["norm"]:
            q, k = lo.rms_norm(q, self.qn, self.eps), lo.rms_norm(k, self.kn, self.eps)
        pos = np.arange(n)
        if m.get("q_temp"):
            q = q * lo.query_temperature(pos, m["q_temp"]["coef"], m["q_temp"]["every"])[:, None]
        q, k, v = q.reshape(n, H, -1), k.reshape(n, G, -1), v.reshape(n, G, -1)
        mask = lo.window_mask(pos, pos, m["mask"]["size"]) if m["mask"]["size"] > 0 else pos[:, None] >= pos[None]
        sl = lo.alibi_slopes(H) if self.flags["bias"] else np.zeros(H)
        out = np.zeros((n, H, m["vdim"]))
        for h in range(H):
            g = h // (H // G)
            sc = lo.distance_bias(q[:, h] @ k[:, g].T * m["scale"], pos, pos, sl[h])
            if self.flags["sink"]:
                p = lo.softmax_with_sink(sc, mask)
            else:
                sc = np.where(mask, sc, -np.inf)
                p = np.exp(sc - sc.max(1, keepdims=True))
                p /= p.sum(1, keepdims=True)
            out[:, h] = p @ v[:, g]
        if self.flags["gate"]:
            out *= (1 / (1 + np.exp(-x[:, -H:])))[:, :, None]
        return out.reshape(n, -1)

    def run(self, portions):
        """portions: steps, each a list of (sequence, first, end). Returns the outputs per sequence; ranges of one token
        go through the decode kernel, longer ones through append + tiles (or everything through the fp32 kernels)."""
        import torch
        pkg, a, ow = self.pkg, self.a, self.m["heads"] * self.m["vdim"]
        got = [np.full((len(x), ow), np.nan) for x in self.rows]
        up = lambda v, t=np.int32: torch.from_numpy(np.ascontiguousarray(v, t)).to(self.dev)
        for step in portions:
            step = sorted(step, key=lambda p: p[2] - p[1] > 1)
            one = sum(e - b == 1 for _, b, e in step)
            x = np.concatenate([self.rows[s][b:e] for s, b, e in step])
            n, ld = len(x), x.shape[1] + 3
            buf = np.zeros((n, ld), np.float32)
            buf[:, :x.shape[1]] = x
            pos = np.concatenate([np.arange(b, e) for _, b, e in step])
            slot = np.concatenate([np.full(e - b, s) for s, b, e in step])
            tiles, at = [], one
            for s, b, e in step[one:]:
                for k in range(0, e - b, 64):
                    tiles.append([at + k, min(64, e - b - k), s, b + k])
                at += e - b
            d, dp, ds, dt = up(buf, np.float32), up(pos), up(slot), up(tiles if tiles else [[0, 0, 0, 0]])
            out = torch.zeros((n, ow + 5), device=self.dev, dtype=torch.float32 if self.f32 else torch.bfloat16)
            L, off = pkg.lib, one * 4
            if self.f32:
                pkg.check(L.cmlb200_qk_norm_append(a, d.data_ptr(), ld, dp.data_ptr(), ds.data_ptr(), n, None))
                pkg.check(L.cmlb200_attention_rows_f32(a, d.data_ptr(), ld, dp.data_ptr(), ds.data_ptr(), n, out.data_ptr(), ow + 5, None))
            else:
                if n > one:
                    pkg.check(L.cmlb200_qk_norm_append(a, d.data_ptr() + one * ld * 4, ld, dp.data_ptr() + off, ds.data_ptr() + off, n - one, None))
                    pkg.check(L.cmlb200_attention_tiles(a, d.data_ptr(), ld, dt.data_ptr(), len(tiles), out.data_ptr(), ow + 5, None))
                if one:
                    keys = max(b for _, b, e in step if e - b == 1)
                    pkg.check(L.cmlb200_attention_one(a, d.data_ptr(), ld, dp.data_ptr(), ds.data_ptr(), one, keys, out.data_ptr(), ow + 5, None))
            torch.cuda.synchronize()
            o, at = out.float().cpu().numpy(), 0
            assert (o[:, ow:] == 0).all()
            for s, b, e in step:
                got[s][b:e] = o[at:at + e - b, :ow]
                at += e - b
        return got


def mixer(H, G, D, V, window, scale=None, coef=0.3, every=11):
    return {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale or D ** -0.5, "mask": {"size": window}, "q_temp": {"coef": coef, "every": every}}


def tol(f32):
    return 2e-5 if f32 else 1.5e-2


def whole(lengths):
    return [[(s, 0, n) for s, n in enumerate(lengths)]]


def token_by_token(lengths):
    return [[(s, t, t + 1) for s, n in enumerate(lengths) if t < n] for t in range(max(lengths))]


SHAPES = [(4, 2, 32, 48, 23), (3, 3, 13, 7, 1), (20, 2, 72, 136, 100), (8, 1, 64, 64, 64), (2, 2, 128, 128, 65), (6, 3, 256, 256, 17), (5, 5, 16, 80, 1000)]


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("shape", SHAPES)
def test_prompts_and_tokens(pkg, torch_dev, shape, f32):
    lengths = [130, 1, 65, 17]
    want = None
    for steps in (whole(lengths), token_by_token(lengths)):
        L = Layer(pkg, torch_dev, mixer(*shape), lengths, f32)
        want = want or [L.want(s) for s in range(len(lengths))]
        for w, g in zip(want, L.run(steps)):
            assert np.abs(w - g).max() < tol(f32) * max(1, np.abs(w).max())


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("off", ["sink", "bias", "gate", "norm", "all"])
def test_each_mechanism_switched_off(pkg, torch_dev, off, f32):
    flags = {k: not (off in (k, "all")) for k in ("sink", "bias", "gate", "norm")}
    m = mixer(6, 2, 48, 32, 0 if off == "all" else 40)
    if off == "all":
        m["q_temp"] = None
    lengths = [150, 90]
    for steps in (whole(lengths), token_by_token(lengths)):
        L = Layer(pkg, torch_dev, m, lengths, f32, **flags)
        for s, g in enumerate(L.run(steps)):
            assert np.abs(L.want(s) - g).max() < tol(f32) * 2


@pytest.mark.parametrize("f32", [False, True])
def test_portions_beside_single_tokens(pkg, torch_dev, f32):
    lengths = [200, 131, 40, 7]
    r = np.random.default_rng(5)
    at, steps = [0] * 4, []
    while any(a < n for a, n in zip(at, lengths)):
        step = []
        for s in range(4):
            k = min(int(r.choice([0, 1, 1, 2, 3, 5, 16, 33, 64, 70])), lengths[s] - at[s])
            if k:
                step.append((s, at[s], at[s] + k))
                at[s] += k
        if step:
            steps.append(step)
    L = Layer(pkg, torch_dev, mixer(4, 2, 24, 40, 37), lengths, f32)
    for s, g in enumerate(L.run(steps)):
        assert np.abs(L.want(s) - g).max() < tol(f32) * 2


def stand_out(L, pairs, strength=12.0):
    """For each (query, key) position of sequence 0: the query points along the key in every head, strongly enough
    that the key, where it is seen, takes nearly all the weight; its value is made large and unlike the others."""
    m = L.m
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    x = L.rows[0]
    r = np.random.default_rng(9)
    for i, (q, k) in enumerate(pairs):
        d = r.choice([-1.0, 1.0], (G, D))
        x[k, L.qw:L.qw + L.kw] = d.ravel()
        x[k, L.qw + L.kw:L.qw + L.kw + L.vw] = 4.0 * r.choice([-1.0, 1.0], L.vw)
        x[q, :L.qw] = np.repeat(d, H // G, 0).ravel()
    L.m["scale"] = L.a.scale = strength * 2 / D


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("window", [16, 17, 31, 33, 64, 80, 129])
def test_window_edges(pkg, torch_dev, window, f32):
    """Keys exactly at the edge: distance window - 1 is seen and dominates, distance window is not and leaves no
    trace. Queries sit around block and tile borders, in prompts and decoded."""
    n = 330
    qs = [q for q in (window - 1, window, 63 + window, 64 + window, 160, 175, 192, 255, 256, 329) if window <= q < n]
    for off in (window - 1, window):
        pairs, used = [], set()
        for q in qs:
            if q - off not in used and q not in used:
                pairs.append((q, q - off))
                used |= {q, q - off}
        for steps in ([[(0, 0, n)]], [[(0, 0, 100)], [(0, 100, 102)], [(0, 102, 163)]] + [[(0, t, t + 1)] for t in range(163, n)]):
            L = Layer(pkg, torch_dev, mixer(4, 2, 32, 16, window, coef=0.1, every=64), [n], f32, bias=False)
            stand_out(L, pairs)
            want, got = L.want(0), L.run(steps)[0]
            assert np.abs(want - got).max() < tol(f32) * 4
            # the inputs do what they are for: moving the edge by one changes those rows beyond the tolerance
            L.m["mask"]["size"] = window + (1 if off == window else -1)
            other = L.want(0)
            rows = [q for q, _ in pairs]
            assert (np.abs(other - want)[rows].max(1) > 10 * tol(f32)).all()


@pytest.mark.parametrize("f32", [False, True])
def test_far_key_among_hundreds(pkg, torch_dev, f32):
    """No window: one key hundreds of tokens back takes the weight, wherever it lies in its block or tile."""
    n = 900
    pairs = [(q, k) for q, k in ((899, 0), (898, 15), (897, 16), (896, 63), (895, 64), (850, 127), (833, 128), (770, 511), (769, 300))]
    for steps in ([[(0, 0, n)]], [[(0, 0, 760)]] + [[(0, t, t + 1)] for t in range(760, n)]):
        L = Layer(pkg, torch_dev, mixer(4, 2, 32, 16, 0, coef=0.0), [n], f32, bias=False, gate=False)
        stand_out(L, pairs)
        want, got = L.want(0), L.run(steps)[0]
        assert np.abs(want - got).max() < tol(f32) * 4
        for q, k in pairs:
            assert np.abs(want[q]).max() > 2


@pytest.mark.parametrize("f32", [False, True])
def test_sink_outweighs_weak_keys(pkg, torch_dev, f32):
    """All scores far below 0: nearly the whole weight goes to the sink, and what is left must be in proportion;
    then far above: the sink must vanish without overflow."""
    n = 80
    for sign in (-1.0, 1.0):
        for steps in ([[(0, 0, n)]], [[(0, t, t + 1)] for t in range(n)]):
            L = Layer(pkg, torch_dev, mixer(4, 2, 32, 16, 30, coef=0.0), [n], f32, bias=False, gate=False, norm=False)
            x = L.rows[0]
            x[:, :L.qw], x[:, L.qw:L.qw + L.kw] = 1.0, sign
            L.m["scale"] = L.a.scale = (3.0 if sign < 0 else 90.0) / 32
            want, got = L.want(0), L.run(steps)[0]
            assert np.abs(want - got).max() < tol(f32)
            if sign < 0:
                t = np.arange(n)
                seen = np.minimum(t + 1, 30) * np.exp(-3.0)
                v = x[:, L.qw + L.kw:L.qw + L.kw + L.vw].reshape(n, 2, 16)
                mean = np.stack([v[max(0, i - 29):i + 1].mean(0) for i in t]).repeat(2, 1).reshape(n, -1)
                assert np.allclose(want, mean * (seen / (1 + seen))[:, None])


def test_long_decode_splits_keys_over_a_cluster(pkg, torch_dev):
    """Few rows and thousands of keys: up to eight CTAs share a row's keys; the split must not show."""
    n = 3000
    for shape in ((4, 1, 64, 64, 0), (2, 2, 128, 96, 2500), (10, 1, 32, 136, 1500)):
        L = Layer(pkg, torch_dev, mixer(*shape, coef=0.1, every=500), [n], False)
        got = L.run([[(0, 0, n - 9)]] + [[(0, t, t + 1)] for t in range(n - 9, n)])[0]
        want = L.want(0)
        assert np.abs(want - got)[-200:].max() < tol(False)


def test_attention_refuses_bad_arguments(pkg, torch_dev):
    L = Layer(pkg, torch_dev, mixer(4, 2, 32, 16, 8), [16], False)
    fake, lib = L.kp.data_ptr(), pkg.lib
    for field, value in (("kv_heads", 3), ("dim_ld", 40), ("vdim_ld", 8), ("block_size", 24), ("cache_dtype", pkg.DT_BF16), ("k_pool", None), ("table_ld", 0)):
        a = pkg.Attn.from_buffer_copy(L.a)
        setattr(a, field, value)
        assert lib.cmlb200_attention_one(a, fake, 256, fake, fake, 1, 1, fake, 64, None) == -1
        assert lib.cmlb200_attention_tiles(a, fake, 256, fake, 1, fake, 64, None) == -1
