"""Kept-window and chunked attention, the gated delta rule, residual streams and grouped routing: each kernel against the
plain restatement (lenedra_oracle.py). Projections are made directly, so that single keys can be made to stand out just
inside and just outside a window, a chunk or the kept tokens, at block borders and far away."""
import numpy as np
import pytest

import lenedra_oracle as lo

pytestmark = pytest.mark.gpu
BS = 16
RNG = lambda s: np.random.default_rng(s)
pad = lambda n, to: (n + to - 1) // to * to


def up(a, dev, dtype=np.float32):
    import torch
    return torch.from_numpy(np.ascontiguousarray(a, dtype)).to(dev)


def bf16(a, dev):
    return up(a, dev).bfloat16()


def sync():
    import torch
    torch.cuda.synchronize()


# ---- attention -----------------------------------------------------------------------------------------------
class Layer:
    """Random projections of `lengths` tokens per sequence, a shuffled block table and device pools.
    kind "kept": keys as values, norms per head, a distance bias, first tokens kept. "chunk": values, a learned sink."""

    def __init__(self, pkg, dev, kind, m, lengths, f32, seed=0, sink=True, factor=1.0):
        import torch
        self.pkg, self.dev, self.kind, self.m, self.f32, self.factor = pkg, dev, kind, m, f32, factor
        H, G, D, V = (m[k] for k in ("heads", "kv_heads", "dim", "vdim"))
        r = RNG(seed)
        self.qw, self.kw, self.vw = H * D, G * D, G * V if kind == "chunk" else 0
        self.rows = [r.standard_normal((n, self.qw + self.kw + self.vw)).astype(np.float32) for n in lengths]
        self.qn, self.kn = ((1 + 0.3 * r.standard_normal(D)).astype(np.float32) for _ in range(2))
        self.sinks = (1 + 2 * r.standard_normal(H)).astype(np.float32) if sink and kind == "chunk" else None
        self.eps = 1e-2
        per = max(pad(n, BS) // BS for n in lengths)
        ids = r.permutation(per * len(lengths) + 3)
        self.table = np.zeros((len(lengths), per + 1), np.int32)
        for s in range(len(lengths)):
            self.table[s, :per] = ids[s * per:(s + 1) * per]
        t = torch.float32 if f32 else torch.float16
        self.kp, self.vp = (torch.full((len(ids) * BS, G, pad(d, 16)), float("nan"), dtype=t, device=dev) for d in (D, V))       # nothing but written slots may be read
        self.keep = [up(self.qn, dev), up(self.kn, dev), up(lo.slopes(H), dev), up(self.table, dev, np.int32), up(self.sinks if self.sinks is not None else [0], dev)]
        k, kept = self.keep, kind == "kept"
        self.a = pkg.Attn(H, G, D, V, pad(D, 16), pad(V, 16), m["scale"], m["mask"]["size"] if kept else 0, k[2].data_ptr() if kept else None, int(self.sinks is not None),
                          k[0].data_ptr() if kept else None, k[1].data_ptr() if kept else None, self.eps, 0, 0, -1, pkg.DT_F32 if f32 else pkg.DT_F16, self.kp.data_ptr(),
                          self.vp.data_ptr(), BS, k[3].data_ptr(), self.table.shape[1], 0, m["mask"].get("keep_first", 0), 0 if kept else m["mask"]["size"],
                          k[4].data_ptr() if self.sinks is not None else None, int(kept), int(kept), 0.0 if factor == 1.0 else factor)

    def want(self, s):
        m, x = self.m, self.rows[s].astype(np.float64)
        n, H, G, D = len(x), m["heads"], m["kv_heads"], m["dim"]
        pos = np.arange(n)
        q, k = x[:, :self.qw].reshape(n, H, D), x[:, self.qw:self.qw + self.kw].reshape(n, G, D)
        if self.kind == "kept":
            v, q, k = k, q / lo.rms(q, self.eps) * self.qn, k / lo.rms(k, self.eps) * self.kn
            o = lo.grouped_attention(q, k, v, lo.window_with_kept(pos, pos, m["mask"]["size"], m["mask"]["keep_first"]), m["scale"], lo.slopes(H), pos[:, None] - pos[None])
        else:
            v = x[:, self.qw + self.kw:].reshape(n, G, -1)
            o = lo.grouped_attention(q, k, v, lo.same_chunk(pos, pos, m["mask"]["size"]), m["scale"], sink=self.sinks)
        return o.reshape(n, -1) * self.factor

    def run(self, steps):
        """steps: lists of (sequence, first, end). Single tokens go through the decode kernel, ranges through append and tiles, or
        everything through the 32-bit kernels."""
        import torch
        pkg, L, a, ow = self.pkg, self.pkg.lib, self.a, self.m["heads"] * self.m["vdim"]
        got = [np.full((len(x), ow), np.nan) for x in self.rows]
        for step in steps:
            step = sorted(step, key=lambda p: p[2] - p[1] > 1)
            one = sum(e - b == 1 for _, b, e in step)
            x = np.concatenate([self.rows[s][b:e] for s, b, e in step])
            n, ld = len(x), x.shape[1] + 3
            buf = np.zeros((n, ld), np.float32)
            buf[:, :x.shape[1]] = x
            tiles, at = [], one
            for s, b, e in step[one:]:
                tiles += [[at + k, min(64, e - b - k), s, b + k] for k in range(0, e - b, 64)]
                at += e - b
            d, dp = up(buf, self.dev), up(np.concatenate([np.arange(b, e) for _, b, e in step]), self.dev, np.int32)
            ds, dt = up(np.concatenate([np.full(e - b, s) for s, b, e in step]), self.dev, np.int32), up(tiles or [[0] * 4], self.dev, np.int32)
            out = torch.zeros((n, ow + 5), device=self.dev, dtype=torch.float32 if self.f32 else torch.bfloat16)
            P = lambda t, k=0: t.data_ptr() + k
            if self.f32:
                pkg.check(L.cmlb200_qk_norm_append(a, P(d), ld, P(dp), P(ds), n, None))
                pkg.check(L.cmlb200_attention_rows_f32(a, P(d), ld, P(dp), P(ds), n, P(out), ow + 5, None))
            else:
                if n > one:
                    pkg.check(L.cmlb200_qk_norm_append(a, P(d, one * ld * 4), ld, P(dp, one * 4), P(ds, one * 4), n - one, None))
                    pkg.check(L.cmlb200_attention_tiles(a, P(d), ld, P(dt), len(tiles), P(out), ow + 5, None))
                if one:
                    pkg.check(L.cmlb200_attention_one(a, P(d), ld, P(dp), P(ds), one, max(b for _, b, e in step if e - b == 1), P(out), ow + 5, None))
            sync()
            o, at = out.float().cpu().numpy(), 0
            assert (o[:, ow:] == 0).all()
            for s, b, e in step:
                got[s][b:e] = o[at:at + e - b, :ow]
                at += e - b
        return got


def kept(H, G, D, size, keep, scale=None):
    return {"heads": H, "kv_heads": G, "dim": D, "vdim": D, "scale": scale or D ** -0.5, "mask": {"size": size, "keep_first": keep}}


def chunk(H, G, D, V, size, scale=None):
    return {"heads": H, "kv_heads": G, "dim": D, "vdim": V, "scale": scale or D ** -0.5, "mask": {"size": size}}


def tol(f32):
    return 2e-5 if f32 else 1.5e-2


def schedules(lengths, seed=3):
    """Whole prompts, single tokens, portions of two and more, and a random mixture."""
    out = [[[(s, 0, n) for s, n in enumerate(lengths)]], [[(s, t, t + 1) for s, n in enumerate(lengths) if t < n] for t in range(max(lengths))],
           [[(s, t, min(t + k, n)) for s, n in enumerate(lengths) if t < n] for k in (2,) for t in range(0, max(lengths), k)]]
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


KEPT = [(4, 2, 32, 23, 5), (3, 3, 13, 1, 9), (20, 2, 72, 100, 0), (8, 1, 64, 64, 16), (2, 2, 128, 65, 70), (6, 3, 200, 17, 33), (5, 5, 16, 1000, 3), (1, 1, 256, 40, 64)]
CHUNK = [(4, 2, 32, 48, 23), (3, 3, 13, 7, 1), (20, 2, 72, 136, 100), (8, 1, 64, 64, 64), (2, 2, 128, 128, 65), (6, 3, 256, 200, 16), (5, 5, 16, 80, 1000)]


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("shape", KEPT + CHUNK)
def test_attention_in_every_schedule(pkg, torch_dev, shape, f32):
    lengths = [150, 1, 65, 17]
    m = kept(*shape) if shape in KEPT else chunk(*shape)
    L = Layer(pkg, torch_dev, "kept" if shape in KEPT else "chunk", m, lengths, f32, factor=1.0 if shape[0] % 2 else -0.7)
    want = [L.want(s) for s in range(len(lengths))]
    for steps in schedules(lengths):
        for w, g in zip(want, L.run(steps)):
            assert np.abs(w - g).max() < tol(f32) * max(1, np.abs(w).max())


@pytest.mark.parametrize("f32", [False, True])
def test_without_a_sink(pkg, torch_dev, f32):
    a, b = (Layer(pkg, torch_dev, "chunk", chunk(6, 2, 48, 32, 40), [90], f32, sink=s) for s in (True, False))
    for L in (a, b):
        for steps in schedules([90]):
            assert np.abs(L.want(0) - L.run(steps)[0]).max() < tol(f32) * 2
    assert np.abs(a.want(0) - b.want(0)).max() > 0.1


@pytest.mark.parametrize("f32", [False, True])
def test_a_large_sink_and_a_tiny_one(pkg, torch_dev, f32):
    """One head's sink takes nearly everything, another's nothing; neither may overflow or vanish early."""
    L = Layer(pkg, torch_dev, "chunk", chunk(4, 2, 16, 16, 30), [70], f32)
    L.sinks = np.array([60.0, -60.0, 5.0, 0.0], np.float32)
    L.keep[4] = up(L.sinks, torch_dev)
    L.a.sinks = L.keep[4].data_ptr()
    want = L.want(0)
    assert np.abs(want[:, :16]).max() < 1e-15 and np.abs(want[:, 16:32]).max() > 1
    for steps in schedules([70]):
        assert np.abs(want - L.run(steps)[0]).max() < tol(f32) * 3


def stand_out(L, pairs):
    """For each (query, key) position of sequence 0 every head's query points along the key, strongly enough that the key
    takes nearly all the weight wherever it is seen (steep heads of a distance bias aside)."""
    m, x, r = L.m, L.rows[0], RNG(9)
    H, G, D = m["heads"], m["kv_heads"], m["dim"]
    for q, k in pairs:
        key = r.choice([-1.0, 1.0], (G, D))
        x[k, L.qw:L.qw + L.kw] = key.ravel()
        x[q, :L.qw] = np.repeat(key, H // G, axis=0).ravel()


def edges(L, f32, n, pairs, move):
    """Outputs agree in prompts, portions and decoding, and `move` (a change of the mask or of the inputs, in the restatement alone)
    would show at every pair's query."""
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
@pytest.mark.parametrize("size", [16, 17, 31, 33, 64, 80, 129])
def test_window_edges(pkg, torch_dev, size, f32):
    """Distance size - 1 is seen, distance size is not; queries sit around block and tile borders."""
    n = 330
    for off, step in ((size - 1, -1), (size, 1)):
        qs = [q for q in (size + 9, size + 10, 63 + size, 64 + size, 160, 175, 192, 255, 256, 329) if q - off > 9]
        L = Layer(pkg, torch_dev, "kept", kept(8, 2, 32, size, 5, 0.7), [n], f32)
        edges(L, f32, n, disjoint([(q, q - off) for q in qs]), lambda: L.m["mask"].update(size=size + step))


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("keep", [1, 6, 15, 16, 17, 40, 64, 70, 128])
def test_first_tokens_are_kept_and_the_next_are_not(pkg, torch_dev, keep, f32):
    """From hundreds of tokens on, the last kept token is seen and the first one behind it is not."""
    n = 330
    for key, step in ((keep - 1, -1), (keep, 1)):
        L = Layer(pkg, torch_dev, "kept", kept(16, 4, 32, 24, keep, 1.2), [n], f32)
        edges(L, f32, n, [(329, key)], lambda: L.m["mask"].update(keep_first=keep + step))
        L = Layer(pkg, torch_dev, "kept", kept(16, 4, 32, 24, keep, 1.2), [n], f32)
        edges(L, f32, n, [(keep + 60, key)], lambda: L.m["mask"].update(keep_first=keep + step))


@pytest.mark.parametrize("f32", [False, True])
def test_tokens_at_the_start_with_more_kept_than_there_are(pkg, torch_dev, f32):
    L = Layer(pkg, torch_dev, "kept", kept(4, 4, 16, 3, 12), [1, 2, 3, 5, 12, 13, 15, 16], f32)
    for steps in schedules([1, 2, 3, 5, 12, 13, 15, 16]):
        for s, g in enumerate(L.run(steps)):
            assert np.abs(L.want(s) - g).max() < tol(f32) * 2


@pytest.mark.parametrize("f32", [False, True])
@pytest.mark.parametrize("size", [16, 17, 31, 48, 64, 70, 128, 200])
def test_chunk_edges(pkg, torch_dev, size, f32):
    """The first key of a query's chunk is seen, the last one of the chunk before is not, from the chunk's first, second and last
    query; chunks begin at position 0 however the prompt is cut."""
    n = 410
    firsts = [c for c in range(size, n, size)]
    inside = disjoint([(c + min(size - 1, n - 1 - c), c) for c in firsts if c + 1 < n])
    L = Layer(pkg, torch_dev, "chunk", chunk(4, 2, 32, 24, size, 0.5), [n], f32)

    def without_the_keys():
        for _, k in inside:
            L.rows[0][k, L.qw:L.qw + L.kw] *= -1
    edges(L, f32, n, inside, without_the_keys)
    for first in (0, 1):
        L = Layer(pkg, torch_dev, "chunk", chunk(4, 2, 32, 24, size, 0.5), [n], f32)
        edges(L, f32, n, disjoint([(c + first, c - 1) for c in firsts if c + 1 < n]), lambda: L.m["mask"].update(size=10 * n))


@pytest.mark.parametrize("f32", [False, True])
def test_far_key_among_hundreds(pkg, torch_dev, f32):
    n = 900
    pairs = [(q, k) for q, k in ((899, 0), (898, 15), (897, 16), (896, 31), (895, 32), (894, 63), (893, 64), (850, 127), (833, 128), (770, 511), (769, 300))]
    L = Layer(pkg, torch_dev, "chunk", chunk(4, 2, 32, 24, 1000, 0.6), [n], f32)
    stand_out(L, pairs)
    want = L.want(0)
    for steps in ([[(0, 0, n)]], [[(0, 0, 740)], [(0, 740, 800)], [(0, 800, n)]], [[(0, 0, 760)]] + [[(0, t, t + 1)] for t in range(760, n)]):
        assert np.abs(want - L.run(steps)[0]).max() < tol(f32) * 3
    for _, k in pairs:
        L.rows[0][k, L.qw:L.qw + L.kw] *= -1
    assert (np.abs(L.want(0) - want)[[q for q, _ in pairs]].max(1) > 20 * tol(f32)).all()


def test_long_decode_splits_keys_over_a_cluster(pkg, torch_dev):
    n = 3000
    for kind, m in (("kept", kept(4, 2, 64, 2500, 40)), ("chunk", chunk(8, 1, 32, 48, 2990)), ("kept", kept(4, 4, 128, 200, 1000))):
        L = Layer(pkg, torch_dev, kind, m, [n], False)
        got = L.run([[(0, 0, n - 20)]] + [[(0, t, t + 1)] for t in range(n - 20, n)])[0]
        assert np.abs(L.want(0) - got)[n - 60:].max() < tol(False)


# ---- gated delta rule ----------------------------------------------------------------------------------------
class DeltaLayer:
    def __init__(self, pkg, dev, shape, lengths, f32, seed=0, a_log=(-4, 1), slots=None, factor=1.0):
        import torch
        self.pkg, self.dev, self.f32, self.factor = pkg, dev, f32, factor
        self.H, self.G, self.D, self.V, self.taps = H, G, D, V, taps = shape
        r = RNG(seed)
        self.ch = 2 * G * D + H * V
        # projections lie behind other columns; decay inputs and gate logits come from the second factors
        self.col = 5
        self.rows = [r.standard_normal((n, self.ch + H)).astype(np.float32) for n in lengths]
        self.dec = [r.standard_normal((n, H * D)).astype(np.float32) for n in lengths]
        self.gate = [r.standard_normal((n, H * V)).astype(np.float32) for n in lengths]
        self.conv = (r.standard_normal((self.ch, taps)) / taps ** 0.5).astype(np.float32)
        self.a_log, self.bias = r.uniform(*a_log, H).astype(np.float32), (r.standard_normal(H * D) - 1).astype(np.float32)
        self.norm, self.eps = (1 + 0.3 * r.standard_normal(V)).astype(np.float32), 1e-3
        n = slots or len(lengths)
        self.state, self.ring = torch.full((n, H, D, pad(V, 4)), float("nan"), device=dev), torch.full((n, taps, self.ch), float("nan"), device=dev)
        self.keep = [up(self.conv.T, dev), up(np.exp(self.a_log), dev), up(self.bias, dev), up(self.norm, dev)]
        self.a = pkg.Delta(H, G, D, V, taps, pad(V, 4), self.col, *(k.data_ptr() for k in self.keep), self.eps, 0.0 if factor == 1.0 else factor, self.state.data_ptr(),
                           self.ring.data_ptr())

    def want(self, s, state=False):
        H, G, D, V = self.H, self.G, self.D, self.V
        x, n = self.rows[s].astype(np.float64), len(self.rows[s])
        y, _ = lo.causal_conv(x[:, :self.ch], self.conv.astype(np.float64), np.zeros((self.taps - 1, self.ch)))
        q, k, v = (p.reshape(n, -1, d) for p, d in zip(np.split(y, [G * D, 2 * G * D], axis=1), (D, D, V)))
        q, k = lo.unit(q) * D ** -0.5, lo.unit(k)
        g = np.exp(-np.exp(self.a_log.astype(np.float64))[:, None] * lo.softplus(self.dec[s].astype(np.float64) + self.bias).reshape(n, H, D))
        beta, S = lo.sigmoid(x[:, self.ch:]), np.zeros((H, D, V))
        o = np.stack([lo.delta_rule(q[:, h // (H // G)], k[:, h // (H // G)], v[:, h], g[:, h], beta[:, h], S[h]) for h in range(H)], 1)
        o = o / lo.rms(o, self.eps) * self.norm * lo.sigmoid(self.gate[s].astype(np.float64)).reshape(n, H, V) * self.factor
        return S if state else o.reshape(n, -1)

    def run(self, steps, slot_of=lambda s: s):
        import torch
        pkg, L, a, ow = self.pkg, self.pkg.lib, self.a, self.H * self.V
        got = [np.full((len(x), ow), np.nan) for x in self.rows]
        for step in steps:
            step = sorted(step, key=lambda p: p[2] - p[1] > 1)
            one = sum(e - b == 1 for _, b, e in step)
            cat = lambda parts, extra, at: up(np.pad(np.concatenate([parts[s][b:e] for s, b, e in step]), ((0, 0), (at, extra))), self.dev)
            odd = 3 if self.D % 4 else 4
            d, dec, gate = cat(self.rows, 2, self.col), cat(self.dec, odd, 0), cat(self.gate, 1, 0)
            n, ld, ldd, ldg = len(d), d.shape[1], dec.shape[1], gate.shape[1]
            dp = up(np.concatenate([np.arange(b, e) for _, b, e in step]), self.dev, np.int32)
            ds = up(np.concatenate([np.full(e - b, slot_of(s)) for s, b, e in step]), self.dev, np.int32)
            runs, at = [], one
            for s, b, e in step[one:]:
                runs.append([at, e - b, slot_of(s), b])
                at += e - b
            out = torch.zeros((n, ow + 3), device=self.dev, dtype=torch.float32 if self.f32 else torch.bfloat16)
            t, P = pkg.DT_F32 if self.f32 else pkg.DT_BF16, lambda x: x.data_ptr()
            if n > one:
                w = torch.full((L.cmlb200_delta_work_floats(a, n - one, len(runs)),), float("nan"), device=self.dev)
                dr = up(runs, self.dev, np.int32)
                pkg.check(L.cmlb200_delta_rows(a, P(d), ld, P(dec), ldd, P(gate), ldg, P(dp), P(ds), one, n - one, P(dr), len(runs), P(w), P(out), t, ow + 3, None))
            if one:
                pkg.check(L.cmlb200_delta_one(a, P(d), ld, P(dec), ldd, P(gate), ldg, P(dp), P(ds), one, P(out), t, ow + 3, None))
            sync()
            o, at = out.float().cpu().numpy(), 0
            assert (o[:, ow:] == 0).all()
            for s, b, e in step:
                got[s][b:e] = o[at:at + e - b, :ow]
                at += e - b
        return got


DELTA = [(4, 2, 32, 48, 4), (3, 3, 13, 7, 3), (6, 1, 72, 136, 2), (2, 2, 64, 64, 5), (2, 1, 128, 128, 4), (1, 1, 256, 256, 4), (9, 3, 5, 200, 1), (4, 4, 136, 20, 8), (40, 8, 16, 16, 4)]
DTOL = {True: 3e-5, False: 1.5e-2}


@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("shape", DELTA)
def test_delta_rule_in_every_schedule(pkg, torch_dev, shape, f32):
    lengths = [150, 1, 65, 17]
    L = DeltaLayer(pkg, torch_dev, shape, lengths, f32, factor=1.0 if shape[0] % 2 else -0.6)
    want = [L.want(s) for s in range(4)]
    for steps in schedules(lengths):
        for w, g in zip(want, L.run(steps)):               # a new run starts at position 0 in slots that hold other states
            assert np.abs(w - g).max() < DTOL[f32] * max(1, np.abs(w).max())


@pytest.mark.parametrize("a_log", [(-9, -8), (3, 4)])
def test_decays_that_keep_or_forget_everything(pkg, torch_dev, a_log):
    L = DeltaLayer(pkg, torch_dev, (4, 2, 24, 32, 4), [200], True, a_log=a_log)
    want, S = L.want(0), L.want(0, state=True)
    for steps in schedules([200]):
        assert np.abs(want - L.run(steps)[0]).max() < 5e-5 * max(1, np.abs(want).max())
        assert np.abs(L.state[0, :, :, :32].cpu().numpy() - S).max() < 5e-5 * max(1, np.abs(S).max())


def test_state_is_carried_over_hundreds_of_tokens_and_slots_are_used_again(pkg, torch_dev):
    """Slow decays: what the first tokens wrote still shows hundreds of tokens on. Then another sequence takes the slot."""
    L = DeltaLayer(pkg, torch_dev, (2, 1, 64, 64, 4), [700, 40], True, a_log=(-7, -6), slots=3)
    want = [L.want(0), L.want(1)]
    other = L.rows[0][:3].copy()
    L.rows[0][:3] *= -1
    assert np.abs(L.want(0)[600:] - want[0][600:]).max() > 1e-3
    L.rows[0][:3] = other
    decoded = [[(0, t, t + 1)] for t in range(5, 700)]
    assert np.abs(L.run([[(0, 0, 5)]] + decoded, lambda s: 2)[0] - want[0]).max() < 2e-4
    assert np.abs(L.run([[(1, 0, 2)], [(1, 2, 3)], [(1, 3, 40)]], lambda s: 2)[1] - want[1]).max() < 5e-5
    assert np.abs(L.run([[(0, 0, 350)], [(0, 350, 352)], [(0, 352, 700)]], lambda s: 0)[0] - want[0]).max() < 2e-4


def test_one_large_write_is_found_again(pkg, torch_dev):
    """A token's value, written under a key of its own, is read back far behind by a query along that key and not otherwise."""
    L = DeltaLayer(pkg, torch_dev, (2, 2, 32, 16, 1), [300], True, a_log=(-12, -11))
    G, D, V, H = 2, 32, 16, 2
    L.conv[:] = 1
    L.keep[0] = up(L.conv.T, torch_dev)
    L.a.conv = L.keep[0].data_ptr()
    x = L.rows[0]
    key = np.zeros((G, D), np.float32)
    key[:, 3] = 30.0
    x[:, G * D:2 * G * D].reshape(300, G, D)[:, :, 3] = -60.0                        # silu makes these nothing
    x[10, G * D:2 * G * D], x[290, :G * D] = key.ravel(), key.ravel()
    x[10, 2 * G * D:2 * G * D + H * V] = 8.0
    x[:, L.ch:] = 3.0
    want = L.want(0)
    for steps in schedules([300])[:1] + [[[(0, 0, 200)]] + [[(0, t, t + 1)] for t in range(200, 300)]]:
        assert np.abs(L.run(steps)[0] - want).max() < 5e-5 * max(1, np.abs(want).max())
    x[10, 2 * G * D:2 * G * D + H * V:2] = -60.0
    assert np.abs(L.want(0)[290] - want[290]).max() > 0.1


# ---- streams -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("f32", [True, False])
@pytest.mark.parametrize("streams,width", [(1, 64), (2, 75), (3, 144), (4, 128), (5, 33), (8, 96), (2, 4096), (4, 1000)])
def test_join(pkg, synth, torch_dev, streams, width, f32):
    import torch
    r, eps, rows = RNG(streams * width), 1e-3, 7
    ex = lambda *s: synth.bf16_round(r.standard_normal(s))[1]
    x, y, w = ex(streams, rows, width), ex(rows, width), 1 + 0.2 * ex(width)
    mix, to, back = ex(streams, streams), ex(streams), ex(streams)
    P = lambda t: t.data_ptr()
    dt, code, tolerance = (torch.float32, pkg.DT_F32, 2e-6) if f32 else (torch.bfloat16, pkg.DT_BF16, 5e-3)
    k = [up(mix, torch_dev), up(to, torch_dev), up(back, torch_dev), up(w, torch_dev)]
    hc = pkg.Streams(streams, P(k[0]), P(k[1]), P(k[2]))
    ldy, ldo = width + (4 if width % 4 == 0 else 1), width + (4 if width % 4 == 0 else 3)
    norm = lambda u: u / lo.rms(u, eps) * w

    def check(got_x, got, want_x, idx=None):
        assert np.abs(got_x.cpu().numpy().transpose(1, 0, 2) - want_x).max() < 1e-5
        if got is not None:
            u = norm(lo.read_streams(want_x, back.astype(np.float64)))
            u = u if idx is None else u[idx]
            assert np.abs(got.float().cpu().numpy()[:, :width] - u).max() < tolerance * np.abs(u).max() and (got[:, width:].float() == 3).all()
    x64, y64 = x.astype(np.float64), y.astype(np.float64)
    # plain rows, with and without a reader
    for reads in (True, False):
        dx, dy = up(x.transpose(1, 0, 2), torch_dev), up(np.pad(y, ((0, 0), (0, ldy - width))), torch_dev)
        out = torch.full((rows, ldo), 3.0, device=torch_dev, dtype=dt)
        pkg.check(pkg.lib.cmlb200_stream_join(hc, P(dx), P(dy), ldy, None, P(k[3]) if reads else None, eps, rows, width, None, P(out) if reads else None, code, ldo, None))
        sync()
        check(dx, out if reads else None, lo.write_streams(x64, mix.astype(np.float64), to.astype(np.float64), y64))
    # a reader alone, of some rows, and the sum of the streams
    idx = np.array([6, 0, 3])
    dx, di = up(x.transpose(1, 0, 2), torch_dev), up(idx, torch_dev, np.int32)
    for hc2, b in ((hc, back), (pkg.Streams(streams, None, None, None), np.ones(streams))):
        out = torch.full((3, ldo), 3.0, device=torch_dev, dtype=dt)
        pkg.check(pkg.lib.cmlb200_stream_join(hc2, P(dx), None, 0, None, P(k[3]), eps, 3, width, P(di), P(out), code, ldo, None))
        sync()
        u = norm(lo.read_streams(x64, np.asarray(b, np.float64)))[idx]
        assert np.abs(out.float().cpu().numpy()[:, :width] - u).max() < tolerance * np.abs(u).max()
    # experts: some pairs point at rows of y, some at the row itself, and another row joins
    top = 3
    pos = r.permutation(rows * top).astype(np.int32)
    pos[[1, 5, 6, 7, 8]] = -1
    wt, yp, add, selfw = ex(rows * top), ex(rows * top, width), ex(rows, width), ex(rows)
    h = ex(rows, width)
    z = h * selfw[:, None] + add + sum((wt.reshape(rows, top)[:, j] * (pos.reshape(rows, top)[:, j] >= 0))[:, None] * yp[pos.reshape(rows, top)[:, j]] for j in range(top))
    t = [up(pos, torch_dev, np.int32), up(wt, torch_dev), up(selfw, torch_dev), up(add, torch_dev), up(np.pad(yp, ((0, 0), (0, ldy - width))), torch_dev)]
    moe = pkg.Moe(4, top, weight=P(t[1]), pos=P(t[0]), identity=2, self=P(t[2]))
    for in_place in (False, True):
        dx = up(x.transpose(1, 0, 2), torch_dev)
        dh = up(np.pad(h, ((0, 0), (0, ldo - width)), constant_values=3), torch_dev).to(dt)
        out = dh if in_place else torch.full((rows, ldo), 3.0, device=torch_dev, dtype=dt)
        j = pkg.Join(pkg.C.pointer(moe), P(dh), P(t[3]), width)
        pkg.check(pkg.lib.cmlb200_stream_join(hc, P(dx), P(t[4]), ldy, j, P(k[3]), eps, rows, width, None, P(out), code, ldo, None))
        sync()
        check(dx, out, lo.write_streams(x64, mix.astype(np.float64), to.astype(np.float64), z.astype(np.float64)))


@pytest.mark.parametrize("rows,width,streams", [(1, 64, 2), (5, 75, 3), (70, 1030, 1), (3, 4096, 4)])
def test_embedding_into_streams(pkg, synth, torch_dev, rows, width, streams):
    import torch
    r = RNG(rows)
    table = synth.bf16_round(r.standard_normal((31, width)))[1]
    tok = r.integers(0, 31, rows)
    for f32 in (True, False):
        d, dt = (up(table, torch_dev), pkg.DT_F32) if f32 else (bf16(table, torch_dev), pkg.DT_BF16)
        x, t = torch.zeros(rows, streams, width, device=torch_dev), up(tok, torch_dev, np.int32)
        pkg.check(pkg.lib.cmlb200_embed_streams(d.data_ptr(), dt, t.data_ptr(), 2.75, streams, rows, width, 31, x.data_ptr(), None))
        sync()
        assert (x.cpu().numpy() == np.float32(2.75) * table[tok][:, None, :]).all()


def test_packed_columns(pkg, torch_dev):
    import torch
    x = RNG(1).standard_normal((9, 301)).astype(np.float32)
    out, d = torch.full((9, 128), 7.0, device=torch_dev).bfloat16(), up(x, torch_dev)
    pkg.check(pkg.lib.cmlb200_pack_columns(d.data_ptr(), 301, 17, 49, 13, 64, 9, out.data_ptr(), 128, None))
    sync()
    assert torch.equal(out[:, :49], d[:, 17:66].bfloat16()) and torch.equal(out[:, 64:77], d[:, 66:79].bfloat16()) and (out[:, 49:64] == 7).all() and (out[:, 77:] == 7).all()
    assert pkg.lib.cmlb200_pack_columns(d.data_ptr(), 301, 17, 49, 13, 40, 9, out.data_ptr(), 128, None) != 0 and pkg.lib.cmlb200_pack_columns(d.data_ptr(), 60, 17, 49, 0, 0, 9, out.data_ptr(), 128, None) != 0


# ---- routing -------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("rows", [1, 2, 31, 32, 33, 300])
@pytest.mark.parametrize("experts,identity,top,groups,keep", [(8, 4, 4, 4, 3), (7, 3, 3, 5, 2), (6, 0, 2, 1, 1), (5, 1, 6, 2, 2), (60, 4, 6, 8, 3), (1, 1, 1, 2, 1), (200, 56, 8, 64, 8),
                                                             (700, 300, 5, 4, 1)])
@pytest.mark.parametrize("align", [1, 128])
def test_choice_within_groups(pkg, torch_dev, rows, experts, identity, top, groups, keep, align):
    import torch
    n, r = experts + identity, RNG(rows + experts)
    z, corr = (r.standard_normal((rows, n)) * 2).astype(np.float32), r.choice([0.3, -0.4, -2.5, 0.0], n).astype(np.float32) + (0.1 * r.standard_normal(n)).astype(np.float32)
    P = lambda t: t.data_ptr()
    i = lambda k: torch.full((k,), -7, device=torch_dev, dtype=torch.int32)
    room = pkg.lib.cmlb200_moe_positions(rows, top, experts, align)
    t = {"ids": i(rows * top), "weight": torch.zeros(rows * top, device=torch_dev), "pos": i(rows * top), "src": i(room), "expert": i(room), "start": i(experts), "count": i(experts),
         "active": i(experts), "num_active": i(1), "tiles": i(4 * (room // 128 + experts + 1)), "num_tiles": i(1), "self": torch.full((rows,), 9.0, device=torch_dev)}
    dz, dc = up(z, torch_dev), up(corr, torch_dev)
    m = pkg.Moe(experts, top, identity=identity, groups=groups, keep=keep, correction=P(dc), normalize=1, scale=1.75, **{k: P(v) for k, v in t.items()})
    pkg.check(pkg.lib.cmlb200_moe_route(m, P(dz), n, rows, align, None))
    sync()
    g = {k: v.cpu().numpy() for k, v in t.items()}
    ids, w = lo.route(z.astype(np.float64), {"router": np.eye(n), "correction": corr.astype(np.float64)},
                      {"groups": {"count": groups, "keep": keep}, "top": top, "scale": 1.75})
    assert (g["ids"].reshape(rows, top) == ids).all()
    assert np.abs(g["weight"].reshape(rows, top) - w).max() < 3e-6
    if identity:
        assert np.abs(g["self"] - np.where(ids >= experts, w, 0).sum(1)).max() < 5e-6
    real = ids.ravel() < experts
    count = np.bincount(ids.ravel()[real], minlength=experts)
    assert (g["count"] == count).all() and (g["pos"][~real] == -1).all()
    pos, mine = g["pos"][real], ids.ravel()[real]
    assert len(set(pos.tolist())) == len(pos) and (g["expert"][pos] == mine).all() and (g["src"][pos] == (np.arange(rows * top) // top)[real]).all()
    start = np.concatenate([[0], np.cumsum((count + align - 1) // align * align)])
    assert (g["start"] == start[:-1]).all() and g["num_active"][0] == (count > 0).sum()


def test_routing_refusals(pkg):
    dummy = {k: 16 for k in ("ids", "weight", "pos", "src", "expert", "start", "count", "active", "num_active", "tiles", "num_tiles", "self")}
    for kw in ({"top": 9}, {"groups": 5, "keep": 1}, {"groups": 4, "keep": 0}, {"groups": 4, "keep": 1, "top": 3}, {"self": 0}, {"identity": -1}):
        a = {"experts": 6, "top": 2, "identity": 2, **dummy, **kw}
        assert pkg.lib.cmlb200_moe_route(pkg.Moe(**a), 16, 8, 4, 1, None) != 0


# ---- products with a bias and a cap ---------------------------------------------------------------------------
@pytest.mark.parametrize("M", [1, 7, 20, 32, 33, 200])
@pytest.mark.parametrize("N,K", [(96, 64), (211, 144), (75, 33), (1030, 300)])
@pytest.mark.parametrize("bias,cap", [(True, 0.0), (False, 2.0), (True, 0.7)])
def test_products_with_bias_and_cap(pkg, synth, torch_dev, M, N, K, bias, cap):
    import torch
    r = RNG(M + N)
    x, w, b = synth.bf16_round(r.standard_normal((M, K)))[1], synth.bf16_round(r.standard_normal((N, K)) / K ** 0.5)[1], r.standard_normal(N).astype(np.float32)
    want = x.astype(np.float64) @ w.T.astype(np.float64) + (b if bias else 0)
    want = cap * np.tanh(want / cap) if cap else want
    ld = pad(K, 64)
    xp, wp = np.zeros((M, ld), np.float32), np.zeros((pad(N, 16), ld), np.float32)
    xp[:, :K], wp[:N, :K] = x, w
    db, L = up(b, torch_dev), pkg.lib
    for form in ["f32"] + (["gemv"] if M <= 32 else []) + ["gemm"]:
        f32 = form == "f32"
        dx, dw = (up(xp, torch_dev), up(wp, torch_dev)) if f32 else (bf16(xp, torch_dev), bf16(wp, torch_dev))
        W = pkg.Dense(pkg.DT_F32 if f32 else pkg.DT_BF16, N, K, ld, dw.data_ptr(), db.data_ptr() if bias else None, cap)
        y = torch.full((M, N + 3), 5.0, device=torch_dev)
        call = {"f32": L.cmlb200_linear_dense_f32, "gemv": L.cmlb200_gemv_dense, "gemm": L.cmlb200_gemm_dense}[form]
        pkg.check(call(W, dx.data_ptr(), ld, M, y.data_ptr(), N + 3, None))
        sync()
        assert np.abs(y.cpu().numpy()[:, :N] - want).max() < 2e-5 and (y[:, N:] == 5).all()
