"""Latent attention over paged caches, polynomial norms and experts: each kernel against the plain restatement
(latent_oracle.py). Projections are made directly, so that single keys can be made to stand out just inside and just
outside a window, at block borders and far away."""
import ctypes as C

import numpy as np
import pytest

import latent_oracle as la
import lm_util

pytestmark = pytest.mark.gpu
BS = 16
RNG = lambda s: np.random.default_rng(s)
pad = lambda n, to: (n + to - 1) // to * to


def up(a, dev, dtype=np.float32):
    import torch
    return torch.from_numpy(np.ascontiguousarray(a, dtype)).to(dev)


def sync():
    import torch
    torch.cuda.synchronize()


def bf16(a, dev):
    return up(a, dev).bfloat16()


class LatentLayer:
    """Random projections of `lengths` tokens per sequence for a mixer, a shuffled block table and a device pool."""

    def __init__(self, pkg, synth, dev, mixer, lengths, f32, gated=True, seed=0):
        """f32: False (fp16 cache, tcgen05 where it fits), "mma" (fp16 cache, the mma.sync form) or True (32-bit)."""
        self.mma, f32 = f32 == "mma", f32 is True
        r = RNG(seed)
        exact = lambda *shape: synth.bf16_round(r.standard_normal(shape))[1]
        self.pkg, self.synth, self.dev, self.m, self.f32, self.gated = pkg, synth, dev, mixer, f32, gated
        H, D, P, V, R = (mixer[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        self.qw, self.kw, self.gw = H * (D + P), R + P, H * V if gated else 0
        # every projection is exact in bfloat16: what the kernels round is their own
        self.rows = [exact(n, self.qw + self.kw + self.gw) for n in lengths]
        self.uk, self.uv = synth.bf16_round(r.standard_normal((H * D, R)) / R ** 0.5)[1], synth.bf16_round(r.standard_normal((H * V, R)) / R ** 0.5)[1]
        self.cn, self.eps = (1 + 0.3 * r.standard_normal(R)).astype(np.float32), 1e-3
        per = max(pad(n, BS) // BS for n in lengths)
        ids = r.permutation(per * len(lengths) + 3)
        self.table = np.zeros((len(lengths), per + 1), np.int32)
        for s in range(len(lengths)):
            self.table[s, :per] = ids[s * per:(s + 1) * per]
        self.blocks = len(ids)

    def upload(self):
        import torch
        pkg, dev, m = self.pkg, self.dev, self.m
        H, D, P, V, R = (m[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
        self.ld, self.ldr = pad(R + P, 16), pad(R, 64)
        f, mul = la.frequencies(m["rot"])
        t = torch.float32 if self.f32 else torch.float16
        self.pool = torch.full((self.blocks * BS, self.ld), float("nan"), dtype=t, device=dev)            # nothing but written slots may be read
        uk = self.uk.reshape(H, D, R).transpose(0, 2, 1)
        if self.f32:
            self.wukt, self.wuv = up(uk, dev), up(self.uv, dev)
        else:
            w = np.zeros((H, pad(R, 16), pad(D, 64)), np.float32)
            w[:, :R, :D] = uk
            self.wukt = bf16(w, dev)
            vp = pad(V, 16)
            w = np.zeros((pad(H * (D + vp), 16), self.ldr), np.float32)
            w[:H * D, :R] = self.uk
            w[H * D:H * (D + vp), :R].reshape(H, vp, R)[:, :V] = self.uv.reshape(H, V, R)
            self.wukv = bf16(w, dev)
            self.dense = pkg.Dense(pkg.DT_BF16, H * (D + vp), R, self.ldr, self.wukv.data_ptr())
            self.wuv = self.wukv[H * D:]
        self.keep = [up(self.cn, dev), up(f, dev), up(self.table, dev, np.int32)]
        k = self.keep
        self.a = pkg.Latent(H, D, P, V, R, self.ld, self.ldr, m["scale"], (m.get("mask") or {}).get("size", 0), k[0].data_ptr(), self.eps, k[1].data_ptr(), mul,
                            self.qw, self.qw + self.kw if self.gated else -1, pkg.DT_F32 if self.f32 else pkg.DT_F16, self.pool.data_ptr(), BS, k[2].data_ptr(),
                            self.table.shape[1], 0 if self.mma else self.blocks)

    def want(self, s):
        m, x = self.m, self.rows[s].astype(np.float64)
        n, H, D = len(x), m["heads"], m["dim"]
        pos = np.arange(n)
        q = x[:, :self.qw].reshape(n, H, -1)
        kv = x[:, self.qw:self.qw + self.kw]
        c, r = la.rms_norm(kv[:, :m["kv_rank"]], self.cn, self.eps), la.rotate(kv[:, m["kv_rank"]:], pos, m["rot"])
        w = {"uk": self.uk.astype(np.float64), "uv": self.uv.astype(np.float64)}
        o = la.attend(q[:, :, :D], la.rotate(q[:, :, D:], pos, m["rot"]), c, r, w, m, pos, pos).reshape(n, -1)
        return o * la.sigmoid(x[:, self.qw + self.kw:]) if self.gated else o

    def run(self, portions):
        """portions: steps, each a list of (sequence, first, end). Ranges of one token and of up to 64 go over the latents,
        longer ones through the expansion (or everything through the 32-bit kernels)."""
        self.upload()
        self.pkg.check(self.pkg.lib.cmlb200_set_attention_latent_form(1 if self.mma else 2))
        try:
            return self._run(portions)
        finally:
            self.pkg.check(self.pkg.lib.cmlb200_set_attention_latent_form(0))

    def _run(self, portions):
        import torch
        pkg, L, a, m = self.pkg, self.pkg.lib, self.a, self.m
        H, V, ow = m["heads"], m["vdim"], m["heads"] * m["vdim"]
        got = [np.full((len(x), ow), np.nan) for x in self.rows]
        kind = lambda n: 0 if n == 1 else (1 if n <= 64 else 2)
        for step in portions:
            step = sorted(step, key=lambda p: kind(p[2] - p[1]))
            x = np.concatenate([self.rows[s][b:e] for s, b, e in step])
            n, ld = len(x), x.shape[1] + 3
            buf = np.zeros((n, ld), np.float32)
            buf[:, :x.shape[1]] = x
            one = sum(e - b == 1 for _, b, e in step)
            near = sum(e - b for _, b, e in step if e - b <= 64)
            tiles, long, at = [[], []], [], 0
            for s, b, e in step:
                if e - b > 1:
                    for k in range(0, e - b, 64):
                        tiles[kind(e - b) - 1].append([at + k, min(64, e - b - k), s, b + k])
                if e - b > 64:
                    long.append((s, b, e))
                at += e - b
            d = up(buf, self.dev)
            dp = up(np.concatenate([np.arange(b, e) for _, b, e in step]), self.dev, np.int32)
            ds = up(np.concatenate([np.full(e - b, s) for s, b, e in step]), self.dev, np.int32)
            out = torch.zeros((n, ow + 5 + ow % 2), device=self.dev, dtype=torch.float32 if self.f32 else torch.bfloat16)
            old, P = out.shape[1], lambda t, k=0: t.data_ptr() + k
            if self.f32:
                kd = m["kv_rank"] + m["rot_dim"]
                q, o = torch.zeros(n, H * kd, device=self.dev), torch.zeros(n, H * m["kv_rank"], device=self.dev)
                pkg.check(L.cmlb200_latent_query_f32(a, P(self.wukt), P(d), ld, P(dp), P(ds), n, P(q), None))
                s1 = pkg.Attn(H, 1, kd, m["kv_rank"], self.ld, self.ld, m["scale"], a.window, None, 0, None, None, 0, 0, 0, -1, pkg.DT_F32, P(self.pool), P(self.pool), BS,
                              a.block_table, a.table_ld)
                pkg.check(L.cmlb200_attention_rows_f32(s1, P(q), H * kd, P(dp), P(ds), n, P(o), H * m["kv_rank"], None))
                pkg.check(L.cmlb200_latent_output_f32(a, P(self.wuv), P(o), P(d), ld, n, P(out), old, None))
            else:
                if near:
                    q = torch.zeros(near, H * self.ld, device=self.dev, dtype=torch.float16)
                    o = torch.zeros(near, H * self.ldr, device=self.dev, dtype=torch.bfloat16)
                    pkg.check(L.cmlb200_latent_query(a, P(self.wukt), P(d), ld, P(dp), P(ds), near, P(q), None))
                    if one:
                        keys = max(b for _, b, e in step if e - b == 1)
                        pkg.check(L.cmlb200_attention_latent(a, P(q), near, P(dp), P(ds), one, keys, None, 0, P(o), None))
                    if tiles[0]:
                        t = up(tiles[0], self.dev, np.int32)
                        pkg.check(L.cmlb200_attention_latent(a, P(q), near, None, None, 0, max(x[3] + x[1] for x in tiles[0]), P(t), len(tiles[0]), P(o), None))
                    pkg.check(L.cmlb200_latent_output(a, P(self.wuv), P(o), P(d), ld, near, P(out), old, None))
                if long:
                    pkg.check(L.cmlb200_latent_append(a, P(d, near * ld * 4), ld, P(dp, near * 4), P(ds, near * 4), n - near, None))
                    keys, at = [], 0
                    for s, b, e in long:
                        lo = (b - a.window + 1 if 0 < a.window <= b else 0) // BS * BS
                        keys.append([s, lo, e - lo, at])
                        at += pad(e - lo, BS)
                    dk, dv = pad(m["dim"] + m["rot_dim"], 16), pad(V, 16)
                    kp, vp = (torch.zeros(at, H, w, device=self.dev, dtype=torch.float16) for w in (dk, dv))
                    c = torch.zeros(at, self.ldr, device=self.dev, dtype=torch.bfloat16)
                    tab = torch.zeros_like(self.keep[2])
                    s2 = pkg.Attn(H, H, m["dim"] + m["rot_dim"], V, dk, dv, m["scale"], a.window, None, 0, None, None, 0, 0, 0, a.gate_col, pkg.DT_F16, P(kp), P(vp), BS,
                                  P(tab), a.table_ld, int(self.gated))
                    pkg.check(L.cmlb200_latent_gather(a, np.ascontiguousarray(keys, np.int32).ctypes.data, len(keys), P(c), s2, None))
                    pkg.check(L.cmlb200_latent_expand(a, self.dense, P(c), at, s2, None))
                    t = up(tiles[1], self.dev, np.int32)
                    pkg.check(L.cmlb200_attention_tiles(s2, P(d), ld, P(t), len(tiles[1]), P(out), old, None))
            sync()
            st = C.c_int(-1)
            pkg.check(L.cmlb200_attention_latent_status(C.byref(st), 1))
            assert st.value == 0
            res, at = out.float().cpu().numpy(), 0
            assert (res[:, ow:] == 0).all()
            for s, b, e in step:
                got[s][b:e] = res[at:at + e - b, :ow]
                at += e - b
        return got


def mixer(H, D, P, V, R, window=0, scaling=None, base=1000.0, scale=None):
    rot = {"base": base, "dims": P}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    m = {"heads": H, "dim": D, "rot_dim": P, "vdim": V, "kv_rank": R, "rot": rot, "scale": scale or (D + P) ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return m


def tol(f32):
    return 2e-5 if f32 is True else 1.5e-2


def whole(lengths):
    return [[(s, 0, n) for s, n in enumerate(lengths)]]


def token_by_token(lengths):
    return [[(s, t, t + 1) for s, n in enumerate(lengths) if t < n] for t in range(max(lengths))]


def near_only(lengths, k=40):
    return [[(s, t, min(t + k, n)) for s, n in enumerate(lengths) if t < n] for t in range(0, max(lengths), k)]


SHAPES = [(4, 32, 16, 48, 80, 23), (3, 13, 6, 7, 21, 1), (20, 72, 64, 136, 300, 100), (40, 16, 2, 24, 129, 0), (2, 128, 64, 128, 512, 0), (70, 8, 8, 8, 40, 65),
          (1, 200, 32, 200, 256, 1000), (5, 24, 24, 33, 16, 31), (17, 64, 32, 64, 128, 64), (6, 32, 96, 24, 500, 70), (33, 64, 64, 40, 512, 129)]


@pytest.mark.parametrize("f32", [False, "mma", True])
@pytest.mark.parametrize("shape", SHAPES)
def test_prompts_portions_and_tokens(pkg, synth, torch_dev, shape, f32):
    lengths = [130, 1, 65, 17]
    L = LatentLayer(pkg, synth, torch_dev, mixer(*shape), lengths, f32)
    want = [L.want(s) for s in range(len(lengths))]
    for steps in (whole(lengths), near_only(lengths), token_by_token(lengths)):
        for w, g in zip(want, L.run(steps)):
            assert np.abs(w - g).max() < tol(f32) * max(1, np.abs(w).max())


@pytest.mark.parametrize("f32", [False, "mma", True])
@pytest.mark.parametrize("scaling", [None, (4.0, 64, 8.0, 1.0), (1.0, 32, 4.0, 0.5), (40.0, 4096, 32.0, 1.0), (2.0, 4, 50.0, 40.0)])
def test_rotation_without_a_gate(pkg, synth, torch_dev, scaling, f32):
    """The rotated part carries nearly the whole score."""
    lengths = [150, 90]
    L = LatentLayer(pkg, synth, torch_dev, mixer(6, 16, 32, 24, 64, 0, scaling, 300.0, 0.4), lengths, f32, gated=False)
    for x in L.rows:
        x[:, :L.qw].reshape(len(x), 6, 48)[:, :, :16] *= 0.125
    want = [L.want(s) for s in range(2)]
    for steps in (whole(lengths), near_only(lengths), token_by_token(lengths)):
        for w, g in zip(want, L.run(steps)):
            assert np.abs(w - g).max() < tol(f32) * 2


@pytest.mark.parametrize("f32", [False, "mma", True])
def test_portions_beside_single_tokens(pkg, synth, torch_dev, f32):
    lengths = [200, 231, 40, 7]
    for seed in (5, 6):
        r = RNG(seed)
        at, steps = [0] * 4, []
        while any(a < n for a, n in zip(at, lengths)):
            step = []
            for s in range(4):
                k = min(int(r.choice([0, 1, 1, 2, 3, 5, 16, 33, 64, 70, 90])), lengths[s] - at[s])
                if k:
                    step.append((s, at[s], at[s] + k))
                    at[s] += k
            if step:
                steps.append(step)
        L = LatentLayer(pkg, synth, torch_dev, mixer(4, 24, 8, 40, 72, 37), lengths, f32, seed=seed)
        for s, g in enumerate(L.run(steps)):
            assert np.abs(L.want(s) - g).max() < tol(f32) * 2


def stand_out(L, pairs, rotated, strength=14.0):
    """For each (query, key) position of sequence 0 every head's query points along the key, in the unrotated or in the
    rotated part, strongly enough that the key takes nearly all the weight where it is seen; its latent is large in no
    way but unlike the others."""
    m, x, r = L.m, L.rows[0], RNG(9)
    H, D, P, R = m["heads"], m["dim"], m["rot_dim"], m["kv_rank"]
    bf = lambda v: L.synth.bf16_round(np.asarray(v, np.float32))[1]
    for q, k in pairs:
        lat = r.choice([-1.0, 1.0], R)
        x[k, L.qw:L.qw + R] = lat
        qq = np.zeros((H, D + P))
        if rotated:
            part = r.choice([-1.0, 1.0], P)
            x[k, L.qw + R:L.qw + L.kw] = part
            rk = la.rotate(part[None], [k], m["rot"])
            qq[:, D:] = la.rotate(rk, [-q], m["rot"]) * strength / (m["scale"] * P)           # turned back by q: after rotation it lies on the key
        else:
            c = la.rms_norm(lat[None], L.cn.astype(np.float64), L.eps)[0]
            key = (L.uk.astype(np.float64) @ c).reshape(H, D)
            qq[:, :D] = key * strength / (m["scale"] * (key * key).sum(1, keepdims=True))
        x[q, :L.qw] = bf(qq.ravel())


@pytest.mark.parametrize("f32", [False, "mma", True])
@pytest.mark.parametrize("window", [16, 17, 31, 33, 64, 80, 129])
def test_window_edges(pkg, synth, torch_dev, window, f32):
    """Keys exactly at the edge: distance window - 1 is seen and dominates, distance window is not and leaves no trace.
    Queries sit around block and tile borders, in prompts (expanded and over the latents) and decoded."""
    n = 330
    qs = [q for q in (window - 1, window, 63 + window, 64 + window, 160, 175, 192, 255, 256, 329) if window <= q < n]
    for off in (window - 1, window):
        pairs, used = [], set()
        for q in qs:
            if q - off not in used and q not in used:
                pairs.append((q, q - off))
                used |= {q, q - off}
        L = LatentLayer(pkg, synth, torch_dev, mixer(4, 32, 16, 16, 64, window), [n], f32, gated=False)
        stand_out(L, pairs, rotated=False)
        want = L.want(0)
        for steps in ([[(0, 0, n)]], [[(0, t, min(t + 57, n))] for t in range(0, n, 57)],
                      [[(0, 0, 100)], [(0, 100, 102)], [(0, 102, 173)]] + [[(0, t, t + 1)] for t in range(173, n)]):
            got = L.run(steps)[0]
            assert np.abs(want - got).max() < tol(f32) * 4
        # the inputs do what they are for: moving the edge by one changes those rows beyond the tolerance
        L.m["mask"]["size"] = window + (1 if off == window else -1)
        other = L.want(0)
        assert (np.abs(other - want)[[q for q, _ in pairs]].max(1) > 6 * tol(f32)).all()


@pytest.mark.parametrize("f32", [False, "mma", True])
@pytest.mark.parametrize("rotated", [False, True])
def test_far_key_among_hundreds(pkg, synth, torch_dev, rotated, f32):
    """No window: one key hundreds of tokens back takes the weight, wherever it lies in its block or tile."""
    n = 900
    pairs = [(q, k) for q, k in ((899, 0), (898, 15), (897, 16), (896, 31), (895, 32), (894, 63), (893, 64), (850, 127), (833, 128), (770, 511), (769, 300))]
    L = LatentLayer(pkg, synth, torch_dev, mixer(4, 32, 16, 16, 64), [n], f32, gated=False)
    stand_out(L, pairs, rotated, 24.0 if rotated else 14.0)
    want = L.want(0)
    for steps in ([[(0, 0, n)]], [[(0, 0, 740)], [(0, 740, 800)], [(0, 800, 860)], [(0, 860, n)]], [[(0, 0, 760)]] + [[(0, t, t + 1)] for t in range(760, n)]):
        got = L.run(steps)[0]
        assert np.abs(want - got).max() < tol(f32) * 4
    for _, k in pairs:                                 # without those keys the rows would be others
        L.rows[0][k, L.qw:L.qw + 64] *= -1
    assert (np.abs(L.want(0) - want)[[q for q, _ in pairs]].max(1) > 20 * tol(f32)).all()


@pytest.mark.parametrize("form", [False, "mma"])
def test_long_decode_splits_keys_over_a_cluster(pkg, synth, torch_dev, form):
    """Few rows and thousands of keys: up to eight CTAs share a row's keys; the split must not show."""
    n = 3000
    for shape in ((4, 32, 16, 24, 64, 0), (2, 128, 64, 64, 512, 2500), (40, 16, 8, 16, 136, 1500)):
        L = LatentLayer(pkg, synth, torch_dev, mixer(*shape, base=1e5), [n], form)
        got = L.run([[(0, 0, n - 9)]] + [[(0, t, t + 1)] for t in range(n - 9, n)])[0]
        rows = slice(n - 40, n)
        assert np.abs(L.want(0) - got)[rows].max() < tol(False)


@pytest.mark.parametrize("form", [False, "mma"])
def test_many_rows_decode_together(pkg, synth, torch_dev, form):
    """Batches above one block of query rows, with histories from none to hundreds of keys."""
    lengths = [1 + (37 * i) % 300 for i in range(75)]
    L = LatentLayer(pkg, synth, torch_dev, mixer(6, 24, 8, 24, 48, 0), lengths, form)
    prompts = [(s, 0, n - 1) for s, n in enumerate(lengths) if n > 1]
    steps = [prompts[i::6] for i in range(6)]                            # at most 16 sequences to an expansion
    got = L.run(steps + [[(s, n - 1, n) for s, n in enumerate(lengths)]])
    for s in range(len(lengths)):
        assert np.abs(L.want(s) - got[s]).max() < tol(False) * 2


def test_latent_kernels_refuse_bad_arguments(pkg, synth, torch_dev):
    L = LatentLayer(pkg, synth, torch_dev, mixer(4, 32, 16, 16, 64, 8), [16], False)
    L.upload()
    fake, lib = L.pool.data_ptr(), pkg.lib
    for field, value in (("heads", 0), ("rot_dim", 15), ("ld", 72), ("ld", 64), ("ld_rank", 32), ("block_size", 24), ("pool", None), ("table_ld", 0), ("c_norm", None)):
        a = pkg.Latent.from_buffer_copy(L.a)
        setattr(a, field, value)
        assert lib.cmlb200_latent_append(a, fake, 400, fake, fake, 1, None) == -1
        assert lib.cmlb200_latent_query(a, fake, fake, 400, fake, fake, 1, fake, None) == -1
    for field, value in (("rank", 513), ("cache_dtype", pkg.DT_F32), ("block_size", 24), ("ld", 72)):
        a = pkg.Latent.from_buffer_copy(L.a)
        setattr(a, field, value)
        assert lib.cmlb200_attention_latent(a, fake, 1, fake, fake, 1, 1, None, 0, fake, None) == -1
    assert lib.cmlb200_latent_append(L.a, fake, 100, fake, fake, 1, None) == -1


def test_rotation_at_far_positions(pkg, synth, torch_dev):
    """Angles are 32-bit: good to position * 2^-24."""
    import torch
    m = mixer(1, 8, 32, 8, 16, 0, None, 1e4)
    L = LatentLayer(pkg, synth, torch_dev, m, [3], True, gated=False)
    L.upload()
    for p in (0, 1, 1000, 100000):
        table = torch.zeros(1, p // BS + 1, dtype=torch.int32, device=torch_dev)
        a = pkg.Latent.from_buffer_copy(L.a)
        a.block_table, a.table_ld = table.data_ptr(), p // BS + 1
        d = up(L.rows[0][:1], torch_dev)
        pos, slot = up([p], torch_dev, np.int32), up([0], torch_dev, np.int32)
        pkg.check(pkg.lib.cmlb200_latent_append(a, d.data_ptr(), d.shape[1], pos.data_ptr(), slot.data_ptr(), 1, None))
        sync()
        x = L.rows[0][:1].astype(np.float64)
        got = L.pool[p % BS].cpu().numpy()
        want = la.rotate(x[:, L.qw + 16:L.qw + 48], [p], m["rot"])[0]
        assert np.abs(got[16:48] - want).max() < 4e-6 + 4 * p * 2.0 ** -24
        assert np.abs(d.cpu().numpy()[0, 8:40] - la.rotate(x[:, 8:40], [p], m["rot"])[0]).max() < 4e-6 + 4 * p * 2.0 ** -24
        assert np.abs(got[:16] - la.rms_norm(x[:, L.qw:L.qw + 16], L.cn, L.eps)[0]).max() < 1e-5


# ---- rows ----------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("ff", [4, 33, 200, 5001, 12288])
@pytest.mark.parametrize("out", ["bf16", "f32"])
def test_poly_norm(pkg, torch_dev, ff, out):
    import torch
    r = RNG(ff)
    for rows, size in ((3, 1.0), (400, 5.0), (2, 1e-3)):
        z, coef, eps = r.standard_normal((rows, ff)).astype(np.float32) * size, np.array([0.7, -0.3, 0.45, 0.2], np.float32), 1e-3
        buf = np.zeros((rows, pad(ff, 16)), np.float32)
        buf[:, :ff] = z
        d, c = up(buf, torch_dev), up(coef, torch_dev)
        f = torch.zeros(rows, pad(ff, 64), device=torch_dev, dtype=torch.bfloat16 if out == "bf16" else torch.float32)
        pkg.check(pkg.lib.cmlb200_poly_norm(d.data_ptr(), buf.shape[1], rows, ff, c.data_ptr(), eps, f.data_ptr(), pkg.DT_BF16 if out == "bf16" else pkg.DT_F32,
                                            f.shape[1], None))
        sync()
        got, want = f.float().cpu().numpy(), la.poly_norm(z.astype(np.float64), coef.astype(np.float64), eps)
        assert (np.abs(got[:, :ff] - want) <= 1e-5 * (1 + np.abs(want)) + (2.0 ** -8 * np.abs(want) if out == "bf16" else 0)).all() and (got[:, ff:] == 0).all()


@pytest.mark.parametrize("dim,ldy,ldo", [(64, 64, 64), (75, 80, 128), (5000, 5008, 5056)])
@pytest.mark.parametrize("out", ["bf16", "f32"])
def test_residual_add_forms(pkg, torch_dev, dim, ldy, ldo, out):
    import torch
    r, rows, top, eps = RNG(dim), 9, 3, 1e-2
    x, w = r.standard_normal((rows, dim)).astype(np.float32), (1 + 0.5 * r.standard_normal(dim)).astype(np.float32)
    y, wt, pos = r.standard_normal((40, ldy)).astype(np.float32), r.random((rows, top)).astype(np.float32), r.permutation(40)[:rows * top].astype(np.int32)
    dy, dw, dwt, dpos = up(y, torch_dev), up(w, torch_dev), up(wt, torch_dev), up(pos, torch_dev, np.int32)
    moe = pkg.Moe(5, top, None, dwt.data_ptr(), dpos.data_ptr())
    for case in ("copy", "post", "add", "parts"):
        dx = up(x, torch_dev)
        o = torch.zeros(rows, ldo, device=torch_dev, dtype=torch.bfloat16 if out == "bf16" else torch.float32)
        pkg.check(pkg.lib.cmlb200_residual_add(dx.data_ptr(), None if case == "copy" else dy.data_ptr(), ldy, moe if case == "parts" else None,
                                               dw.data_ptr() if case in ("post", "parts") else None, eps, rows, dim, o.data_ptr(),
                                               pkg.DT_BF16 if out == "bf16" else pkg.DT_F32, ldo, None))
        sync()
        Y = y.astype(np.float64)[:rows, :dim]
        if case == "parts":
            Y = (y.astype(np.float64)[pos.reshape(rows, top), :dim] * wt[:, :, None]).sum(1)
        want = x + {"copy": 0 * Y, "add": Y}.get(case, la.rms_norm(Y, w, eps))
        got = o.float().cpu().numpy()
        assert np.abs(dx.cpu().numpy() - want).max() < 1e-5
        assert (np.abs(got[:, :dim] - want) <= 1e-5 + (2.0 ** -8 * np.abs(want) if out == "bf16" else 0)).all() and (got[:, dim:] == 0).all()


# ---- experts -------------------------------------------------------------------------------------------------
class Plan:
    def __init__(self, pkg, dev, rows, experts, top, align):
        import torch
        n = pkg.lib.cmlb200_moe_positions(rows, top, experts, align)
        i = lambda k: torch.full((k,), -1, device=dev, dtype=torch.int32)
        self.t = {"ids": i(rows * top), "weight": torch.zeros(rows * top, device=dev), "pos": i(rows * top), "src": i(n), "expert": i(n), "start": i(experts),
                  "count": i(experts), "active": i(experts), "num_active": i(1), "tiles": i(4 * (n // 128 + experts + 1)), "num_tiles": i(1)}
        self.m = pkg.Moe(experts, top, **{k: v.data_ptr() for k, v in self.t.items()})
        self.n, self.experts, self.top, self.align = n, experts, top, align

    def __getitem__(self, k):
        return self.t[k].cpu().numpy()


@pytest.mark.parametrize("rows", [1, 2, 31, 32, 33, 500])
@pytest.mark.parametrize("experts,top", [(1, 1), (5, 2), (8, 8), (40, 3), (160, 6), (1024, 4)])
@pytest.mark.parametrize("align", [1, 128])
def test_route_and_plan(pkg, torch_dev, rows, experts, top, align):
    r = RNG(rows + experts)
    z = r.standard_normal((rows, experts)).astype(np.float32) * 3
    if rows > 1 and experts > 4:
        z[1] = np.round(z[1])                          # ties
        z[0, :] = 0.25
    buf = np.full((rows, experts + 3), 1e9, np.float32)
    buf[:, :experts] = z
    d, p = up(buf, torch_dev), Plan(pkg, torch_dev, rows, experts, top, align)
    pkg.check(pkg.lib.cmlb200_moe_route(p.m, d.data_ptr(), experts + 3, rows, align, None))
    sync()
    ids, w = la.route(z.astype(np.float64), np.eye(experts), top)
    assert (p["ids"].reshape(rows, top) == ids).all() and np.abs(p["weight"].reshape(rows, top) - w).max() < 1e-6
    count = np.bincount(ids.ravel(), minlength=experts)
    assert (p["count"] == count).all()
    start = np.concatenate([[0], np.cumsum((count + align - 1) // align * align)])
    assert (p["start"] == start[:-1]).all() and start[-1] <= p.n
    pos = p["pos"]
    assert len(set(pos.tolist())) == len(pos)
    assert (p["src"][pos] == np.arange(rows * top) // top).all() and (p["expert"][pos] == ids.ravel()).all()
    assert ((pos >= start[ids.ravel()]) & (pos < start[ids.ravel()] + count[ids.ravel()])).all()
    act = np.nonzero(count)[0]
    assert p["num_active"][0] == len(act) and (p["active"][:len(act)] == act).all()
    tiles = [[start[e] + 128 * i, e, min(128, count[e] - 128 * i), 0] for e in act for i in range((count[e] + 127) // 128)]
    assert p["num_tiles"][0] == len(tiles) and (p["tiles"].reshape(-1, 4)[:len(tiles)] == tiles).all()


@pytest.mark.parametrize("rows", [1, 7, 20, 32, 33, 300])
@pytest.mark.parametrize("experts,top,ff,width", [(5, 2, 40, 144), (3, 3, 17, 75), (1, 1, 64, 64), (40, 3, 48, 192), (9, 4, 330, 700)])
def test_expert_products(pkg, synth, torch_dev, rows, experts, top, ff, width):
    """Both products and the activation of every chosen expert, decode and prompt form and 32-bit, against the restatement."""
    import torch
    r, limit, L = RNG(rows + experts), 0.8, pkg.lib
    ex = lambda *s: synth.bf16_round(r.standard_normal(s))[1]
    x = ex(rows, width)
    g, u, dn = ex(experts, ff, width) / 8, ex(experts, ff, width) / 8, ex(experts, width, ff) / 8
    z = r.standard_normal((rows, experts)).astype(np.float32)
    ids, _ = la.route(z.astype(np.float64), np.eye(experts), top)
    f16, w16 = pad(ff, 16), pad(width, 16)
    gu, dd = np.zeros((experts, 2 * f16, pad(width, 64)), np.float32), np.zeros((experts, w16, pad(ff, 64)), np.float32)
    c = np.arange(ff) // 16 * 32 + np.arange(ff) % 16
    gu[:, c, :width], gu[:, c + 16, :width], dd[:, :width, :ff] = g, u, dn
    x64, ldx, ldf = x.astype(np.float64), pad(width, 64), pad(ff, 64)
    for form in ["f32"] + (["gemv"] if rows <= 32 else []) + ["gemm"]:
        align = 128 if form == "gemm" else 1
        p, dl = Plan(pkg, torch_dev, rows, experts, top, align), up(z, torch_dev)
        pkg.check(L.cmlb200_moe_route(p.m, dl.data_ptr(), experts, rows, align, None))
        f32 = form == "f32"
        put = (lambda a: up(a, torch_dev)) if f32 else (lambda a: bf16(a, torch_dev))
        dt = torch.float32 if f32 else torch.bfloat16
        xs = np.zeros((rows, ldx), np.float32)
        xs[:, :width] = x
        dx, dgu, ddd = put(xs), put(gu), put(dd)
        W1 = pkg.Dense(pkg.DT_F32 if f32 else pkg.DT_BF16, experts * 2 * f16, width, ldx, dgu.data_ptr())
        W2 = pkg.Dense(pkg.DT_F32 if f32 else pkg.DT_BF16, experts * w16, ff, ldf, ddd.data_ptr())
        f, y = torch.zeros(p.n, ldf, device=torch_dev, dtype=dt), torch.full((p.n, width + 4), 7.0, device=torch_dev)
        if f32:
            mid = torch.zeros(p.n, 2 * f16, device=torch_dev)
            pkg.check(L.cmlb200_moe_linear_f32(p.m, W1, dx.data_ptr(), ldx, 1, rows, 2 * f16, mid.data_ptr(), 2 * f16, None))
            pkg.check(L.cmlb200_moe_glu_rows_f32(mid.data_ptr(), 2 * f16, p.n, ff, pkg.ACT_CLAMPED, limit, f.data_ptr(), ldf, None))
            pkg.check(L.cmlb200_moe_linear_f32(p.m, W2, f.data_ptr(), ldf, 0, rows, width, y.data_ptr(), width + 4, None))
        elif form == "gemv":
            pkg.check(L.cmlb200_moe_gemv_glu(p.m, W1, dx.data_ptr(), ldx, 1, rows, ff, pkg.ACT_CLAMPED, limit, f.data_ptr(), ldf, None))
            pkg.check(L.cmlb200_moe_gemv(p.m, W2, f.data_ptr(), ldf, 0, rows, width, y.data_ptr(), width + 4, None))
        else:
            xp = torch.zeros(p.n, ldx, device=torch_dev, dtype=dt)
            pkg.check(L.cmlb200_moe_gather(p.m, dx.data_ptr(), ldx, rows, width, xp.data_ptr(), ldx, None))
            pkg.check(L.cmlb200_moe_gemm_glu(p.m, W1, xp.data_ptr(), ldx, rows, ff, pkg.ACT_CLAMPED, limit, f.data_ptr(), ldf, None))
            pkg.check(L.cmlb200_moe_gemm(p.m, W2, f.data_ptr(), ldf, rows, width, y.data_ptr(), width + 4, None))
            st = C.c_int(-1)
            pkg.check(L.cmlb200_gemm_dense_status(C.byref(st), 1))
            assert st.value == 0
        sync()
        got, pos = y.cpu().numpy(), p["pos"].reshape(rows, top)
        worst, size = 0.0, 0.0
        for row in range(rows):
            for k in range(top):
                e = ids[row, k]
                want = la.clamped_glu(g[e].astype(np.float64) @ x64[row], u[e].astype(np.float64) @ x64[row], limit) @ dn[e].T.astype(np.float64)
                worst, size = max(worst, np.abs(got[pos[row, k], :width] - want).max()), max(size, np.abs(want).max())
        assert worst < (3e-6 if f32 else 8e-3) * size
        assert (got[:, width:] == 7).all()


def test_long_portion_without_room_to_expand(pkg, synth, tmp_path, torch_dev, monkeypatch):
    """A portion whose keys the scratch cache can not take runs over the latents, tiles at a time."""
    monkeypatch.setenv("CMLB200_EXPAND_KEYS", "128")
    cfg, w, folder = lm_util.build(synth, tmp_path, "latent")
    m = pkg.LanguageModel(folder, pkg.DTYPE_BFLOAT16, max_tokens=1024, max_sequences=2)
    t = [RNG(i).integers(0, cfg["vocab"], 420) for i in range(2)]
    a, b = m.open(), m.open()
    got = [[x] for x in m.step([(a, t[0][:250], None), (b, t[1][:70], None)])]       # one fits, the other does not
    for k, x in enumerate(m.step([(a, t[0][250:], None), (b, t[1][70:420], None)])):
        got[k].append(x)
    m.close()
    for k in range(2):
        assert lm_util.error(np.concatenate(got[k]), lm_util.reference(cfg, w, t[k])) < lm_util.TOL[6]
