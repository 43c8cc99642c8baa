"""Throughput of models whose sublayers join side by side through gates, whose layers may loop, and whose mixers are heads that mix their
scores, latents with queried heads, and windowed heads beside a minimal gated recurrence (`python bench.py --loops`), beside the
framework's closest models at equal layer sizes, and every kernel against its roofline with the like kernel of those models
under it. Random weights; layers (and experts) share bytes on disk and are separate copies on the device. Not part of the
default workload."""
import ctypes as C
import json

import numpy as np

import bench_latent
import bench_streams
from bench_layered import NEW, PROMPTS, Timer, copies_for, layered_leg, model_leg

BATCHES = (1, 8, 32)
SIZES = dict(vocab=32000, width=4096, heads=32, kv_heads=32, dim=128, window=1024, taps=3, q_rank=1536, kv_rank=512, rot=64, left=(16, 4, 128, 128, 1024), recurrent=4096, experts=8, top=2,
             expert_ff=8192, groups=(2, 1), loop=(0, 2, 2), layers=6, batches=BATCHES)
EXPERTS = dict(SIZES, width=2048, heads=16, kv_heads=16, q_rank=1024, left=(8, 2, 128, 128, 1024), recurrent=2048, experts=64, top=6, expert_ff=1408, groups=(8, 4))


def config(synth, c):
    """Talking heads and latents, which loop, then windowed heads beside the recurrence."""
    mlp = synth.sigmoid_mlp(c["experts"], c["top"], c["expert_ff"], c["groups"])
    layers = [synth.talking_layer(c["heads"], c["kv_heads"], c["dim"], c["dim"], c["window"], c["taps"], 30.0, mlp, (c["dim"], 1e6), (4.0, 1.0, 4.0, 1024)),
              synth.queried_layer(c["heads"], c["dim"], c["rot"], c["dim"], c["q_rank"], c["kv_rank"], mlp)]
    layers += [synth.recurrent_layer(c["left"], (64, 1e6), c["recurrent"], mlp, 4.0) for _ in range(c["layers"] - 2)]
    return synth.looped_config(c["vocab"], c["width"], layers, c["loop"])


def leg(pkg, synth, torch, c, peaks):
    cfg, W, body, cache, state, moe = config(synth, c), c["width"], 0, 0, 0, 0
    a, b, times = c["loop"]
    for i, layer in enumerate(cfg["layers"]):
        m, runs = layer["mixer"], times if a <= i < b else 1
        moe += runs
        body += runs * (2 * W * W + W * c["experts"])
        if layer["type"] == "attention":
            body += runs * W * c["dim"] * 2 * (c["heads"] + c["kv_heads"])
            cache += runs * 4 * c["kv_heads"] * c["dim"]
        elif layer["type"] == "latent_attention":
            H, D, R, Q, P = c["heads"], c["dim"], c["kv_rank"], c["q_rank"], c["rot"]
            body += runs * (W * (Q + R + P + H) + Q * H * (D + P) + 2 * H * D * R + W * H * D)
            cache += runs * 2 * (R + P)
        else:
            H, G, D, V, _ = c["left"]
            body += runs * (W * (H * (D + V + 1) + G * (D + V)) + 4 * W * c["recurrent"])
            cache += runs * 2 * G * (D + V)
            state += runs * 8 * c["recurrent"]
    E, top, per = c["experts"], c["top"], 2 * W * c["expert_ff"]
    chosen = lambda B: E * (1 - (1 - top / E) ** B)                      # expected number of different experts of a step
    return model_leg(pkg, synth, torch, cfg, c, peaks, body + moe * per * top, lambda B: body + moe * per * chosen(B) + c["vocab"] * W, lambda: cache, state, synth.gated_weight)


# ---- kernels -------------------------------------------------------------------------------------------------
def kernel_table(pkg, torch, peaks):
    T, out = Timer(torch), []
    props = torch.cuda.get_device_properties(0)
    fp32 = props.multi_processor_count * 128 * 2 * peaks.get("sm_max_mhz", 1965.0) / 1e6        # TFLOP/s of the fp32 units at the highest clock: nominal, not measured

    def add(kernel, shape, us, nbytes=0.0, flops=0.0, flops32=0.0):
        """The roofline of a launch is the slowest of its bytes and its operations."""
        t = {"hbm": nbytes / peaks["hbm_gbs"] / 1e3, "tensor": flops / peaks["bf16_tflops"] / 1e6, "fp32": flops32 / fp32 / 1e6}
        bound = max(t, key=t.get)
        out.append({"kernel": kernel, "shape": shape, "us": round(us, 2), "bound": bound, "frac": round(t[bound] / us, 4)})

    for part in (decode_heads, prompt_heads, latents, recurrence, joins, routing, experts):
        part(pkg, torch, T, add)
        torch.cuda.empty_cache()
    return out


P = lambda t, k=0: t.data_ptr() + k


def descriptor(pkg, torch, kind, H, G, D, k, v, table, per, keep, window, slots):
    """kind: "talk", "turn" (rotated windowed heads with a gate), "like" (the grouped layered design)."""
    dev, ch = k.device, (H + 2 * G) * D
    t = [torch.rand(D // 2, device=dev), torch.rand(3, ch, device=dev), torch.randn(slots, 3, ch, device=dev), torch.randn(H, H, device=dev) / H, torch.rand(H, device=dev),
         torch.ones(H * D, device=dev)]
    keep.append(t)
    pools = (pkg.DT_F16, P(k), P(v), 16, P(table), per)
    if kind == "like":
        return pkg.Attn(H, G, D, D, D, D, D ** -0.5, window, P(t[4]), 1, P(t[5]), P(t[5]), 1e-5, 0.1, 512.0, ch, *pools)
    a = pkg.Attn(H, G, D, D, D, D, D ** -0.5, window, None, int(kind == "talk"), None, None, 0, 0, 0, ch if kind == "turn" else -1, *pools)
    a.freq, a.rot_dims = P(t[0]), D if kind == "talk" else D // 2
    if kind == "talk":
        a.taps, a.conv, a.ring, a.cap, a.talk = 3, P(t[1]), P(t[2]), 30.0, P(t[3])
    return a


def decode_heads(pkg, torch, T, add):
    """Decoded tokens behind 1,024 tokens of a window."""
    dev, lib, ck, D, ctx, window = torch.device("cuda:0"), pkg.lib, pkg.check, 128, 4095, 1024
    for B in BATCHES:
        for H, G in ((32, 32), (16, 16), (16, 4), (64, 8)):
            per, keep = ctx // 16 + 1, []
            n = min(24, copies_for(4 * B * window * G * D))
            while n > 1 and n * B * per * 16 * G * D * 4 > 24e9:
                n -= 1
            table = torch.arange(B * per, device=dev, dtype=torch.int32).view(B, per).contiguous()
            pools = [(torch.randn(B * per * 16, G, D, device=dev, dtype=torch.float16), torch.randn(B * per * 16, G, D, device=dev, dtype=torch.float16)) for _ in range(n)]
            ld = (H + 2 * G) * D + H
            qkv, o = torch.randn(B, ld, device=dev), torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
            pos, slot = torch.full((B,), ctx, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32)
            q, sc, sl = torch.randn(B, H, D, device=dev).half(), torch.empty(B, H, 1152, device=dev), 1152
            made = lambda kind: [descriptor(pkg, torch, kind, H, G, D, k, v, table, per, keep, window, B) for k, v in pools]
            scored = lambda a: (lambda b: (setattr(b, "scores", P(sc)), setattr(b, "scores_ld", sl), b)[2])(pkg.Attn.from_buffer_copy(a))
            talk = [(a, scored(a)) for a in made("talk")]
            nbytes, flops, shape = 4.0 * B * window * G * D, 4.0 * B * H * window * D, f"H={H} G={G} B={B} window={window}"
            turn = lambda s, a: ck(lib.cmlb200_rotate_append(a, P(qkv), ld, P(pos), P(slot), 0, B, B, P(q), s))
            score = lambda s, a: ck(lib.cmlb200_talk_scores_rows(a, P(q), P(pos), P(slot), B, window, P(sc), sl, s))
            value = lambda s, b: ck(lib.cmlb200_attention_one(b, P(qkv), ld, P(pos), P(slot), B, ctx, P(o), H * D, s))
            cols = (H + 2 * G) * D
            add("rotate_append (taps)", shape, T.us([lambda s, a=a: turn(s, a) for a, _ in talk], 8), B * (16.0 * cols + 2 * cols) + 12 * cols)
            add("talk_scores_rows", shape, T.us([lambda s, a=a: score(s, a) for a, _ in talk], 8), nbytes / 2, flops / 2, 2.0 * B * window * H * H)
            add("attention_one (given scores)", shape, T.us([lambda s, b=b: value(s, b) for _, b in talk], 8), nbytes / 2, flops / 2)
            add("talking heads, all three", shape, T.us([lambda s, a=a, b=b: (turn(s, a), score(s, a), value(s, b)) for a, b in talk], 8), nbytes, flops, 2.0 * B * window * H * H)
            for kind, name in (("turn", "attention_one (rotated)"), ("like", "  like: attention_one")):
                add(name, shape, T.us([lambda s, a=a: ck(lib.cmlb200_attention_one(a, P(qkv), ld, P(pos), P(slot), B, ctx, P(o), H * D, s)) for a in made(kind)], 8), nbytes, flops)
            del pools, talk
            torch.cuda.empty_cache()


def prompt_heads(pkg, torch, T, add):
    dev, lib, ck, D = torch.device("cuda:0"), pkg.lib, pkg.check, 128
    for n in PROMPTS:
        for H, G, window in ((32, 32, 1024), (16, 16, 1024), (64, 8, 1024), (32, 32, 256)):
            per, keep = n // 16 + 1, []
            table = torch.arange(per, device=dev, dtype=torch.int32).view(1, per).contiguous()
            k, v = torch.randn(per * 16, G, D, device=dev).half(), torch.randn(per * 16, G, D, device=dev).half()
            a, turned, like = (descriptor(pkg, torch, kind, H, G, D, k, v, table, per, keep, window, 1) for kind in ("talk", "turn", "like"))
            ld = (H + 2 * G) * D + H
            qkv, o, q = torch.randn(n, ld, device=dev), torch.empty(n, H * D, device=dev, dtype=torch.bfloat16), torch.randn(n, H, D, device=dev).half()
            tiles = torch.tensor([[i, 64, 0, i] for i in range(0, n, 64)], device=dev, dtype=torch.int32)
            pos, slot = torch.arange(n, device=dev, dtype=torch.int32), torch.zeros(n, device=dev, dtype=torch.int32)
            sl = (min(window + 79, n) + 63) // 64 * 64
            at_once = min(len(tiles), max(1, (192 << 20) // (4 * H * 64 * sl)))
            sc = torch.empty(at_once, H, 64, sl, device=dev)
            b = pkg.Attn.from_buffer_copy(a)
            b.scores, b.scores_ld = P(sc), sl
            pairs, shape = float(np.minimum(np.arange(n) + 1, window).sum()), f"H={H} G={G} rows={n} window={window}"
            parts = [(t, min(at_once, len(tiles) - t)) for t in range(0, len(tiles), at_once)]
            score = lambda s, t, m: ck(lib.cmlb200_talk_scores_tiles(a, P(q), P(tiles, 16 * t), m, n, P(sc), sl, s))
            value = lambda s, t, m: ck(lib.cmlb200_attention_tiles(b, P(qkv), ld, P(tiles, 16 * t), m, P(o), H * D, s))
            us1 = T.us([lambda s: [score(s, t, m) for t, m in parts]], 10)
            add("talk_scores_tiles", shape, us1, 0, 2.0 * pairs * H * D, 2.0 * pairs * H * H)
            us2 = T.us([lambda s: [value(s, t, m) for t, m in parts]], 10)
            add("attention_tiles (given scores)", shape, us2, 0, 2.0 * pairs * H * D)
            us = T.us([lambda s: [(score(s, t, m), value(s, t, m)) for t, m in parts]], 10)
            add("talking heads, both", shape, us, 0, 4.0 * pairs * H * D, 2.0 * pairs * H * H)
            for name, x in (("attention_tiles (rotated)", turned), ("  like: attention_tiles", like)):
                add(name, shape, T.us([lambda s, x=x: ck(lib.cmlb200_attention_tiles(x, P(qkv), ld, P(tiles), len(tiles), P(o), H * D, s))], 10), 0, 4.0 * pairs * H * D)
            if window == 1024:
                cols = (H + 2 * G) * D
                nbytes = n * (4.0 * cols + 2 * cols)
                add("rotate_append (taps)", shape, T.us([lambda s: ck(lib.cmlb200_rotate_append(a, P(qkv), ld, P(pos), P(slot), 0, n, 0, P(q), s))], 10), nbytes)
                add("rotate_append", shape, T.us([lambda s: ck(lib.cmlb200_rotate_append(turned, P(qkv), ld, P(pos), P(slot), 0, n, 0, None, s))], 10), nbytes + n * 2.0 * H * D)
                add("  like: qk_norm_append", shape, T.us([lambda s: ck(lib.cmlb200_qk_norm_append(like, P(qkv), ld, P(pos), P(slot), n, s))], 10), nbytes + n * 2.0 * H * D)


def latents(pkg, torch, T, add):
    """Sinks and a gate per head beside the same without; the queries' second factor beside a product of that size."""
    dev, lib, ck, R, rot = torch.device("cuda:0"), pkg.lib, pkg.check, 512, 64
    for B in BATCHES:
        for H in (16, 32):
            ctx, n = 1024, min(24, copies_for(B * 1024 * (R + rot) * 2))
            ls, sinks = [bench_latent.latent(pkg, torch, H, B, ctx) for _ in range(n)], torch.randn(H, device=dev)
            q, o = torch.randn(B, H, ls[0][0].ld, device=dev).half(), torch.zeros(B, H, R, device=dev).bfloat16()
            pos, slot = torch.full((B,), ctx, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32)
            for name in ("  like: attention_latent", "attention_latent (sinks)"):
                for a, *_ in ls:
                    a.sinks = P(sinks) if name[0] == "a" else None
                calls = [lambda s, a=l[0]: ck(lib.cmlb200_attention_latent(a, P(q), B, P(pos), P(slot), B, ctx, None, 0, P(o), s)) for l in ls]
                add(name, f"H={H} B={B} ctx={ctx}", T.us(calls, 8), 2.0 * B * ctx * (R + rot) + 2.0 * B * H * (2 * R + rot), 2.0 * B * H * ctx * (2 * R + rot))
    for rows in (1, 32, 512, 2048):
        x, w, o = torch.randn(rows, 12000, device=dev), torch.ones(1536, device=dev), torch.empty(rows, 1536, device=dev, dtype=torch.bfloat16)
        add("norm_columns", f"{rows}x1536", T.us([lambda s: ck(lib.cmlb200_norm_columns(P(x), 12000, 6144, 1536, P(w), 1e-5, rows, P(o), pkg.DT_BF16, 1536, s))], 10), rows * 1536 * 6.0)
        x1 = torch.randn(rows, 1536, device=dev)
        add("  like: residual_norm, norm alone", f"{rows}x1536",
            T.us([lambda s: ck(lib.cmlb200_residual_norm(P(x1), None, 0, None, P(w), 1e-5, rows, 1536, None, P(o), pkg.DT_BF16, 1536, s))], 10), rows * 1536 * 6.0)


def recurrence(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    for W in (2048, 4096):
        for B in BATCHES:
            n = 64
            ls = [torch.randn(B, W, device=dev) for _ in range(n)]
            proj, o = torch.randn(B, 3 * W, device=dev), torch.empty(B, W, device=dev, dtype=torch.bfloat16)
            pos, slot = torch.full((B,), 99, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32)
            calls = [lambda s, a=pkg.Gru(W, 0, P(l)): ck(lib.cmlb200_gru_one(a, P(proj), 3 * W, P(pos), P(slot), B, P(o), pkg.DT_BF16, W, s)) for l in ls]
            add("gru_one", f"width={W} B={B}", T.us(calls, 4), B * W * (12.0 + 8 + 2))
        for seqs, rows in ((1, 64), (1, 512), (1, 2048), (4, 512)):
            state, proj, o = torch.randn(seqs, W, device=dev), torch.randn(seqs * rows, 3 * W, device=dev), torch.empty(seqs * rows, W, device=dev, dtype=torch.bfloat16)
            runs, a = torch.tensor([[i * rows, rows, i, 0] for i in range(seqs)], device=dev, dtype=torch.int32), pkg.Gru(W, 0, P(state))
            add("gru_rows", f"width={W} {seqs} x {rows} rows", T.us([lambda s: ck(lib.cmlb200_gru_rows(a, P(proj), 3 * W, P(runs), seqs, P(o), pkg.DT_BF16, W, s))], 10), seqs * rows * W * 14.0)
    bench_streams.delta(pkg, torch, T, lambda kernel, *rest, **kw: add("  like: " + kernel, *rest, **kw))


def joins(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    for rows, W in ((1, 4096), (8, 4096), (32, 4096), (512, 4096), (2048, 4096)):
        n = min(copies_for(rows * W * 30), 64)
        xs = [torch.randn(rows, W, device=dev) for _ in range(n)]
        a, b, h, w, gates = torch.randn(rows, W, device=dev), torch.randn(rows, W, device=dev), torch.empty(rows, W, device=dev, dtype=torch.bfloat16), torch.ones(W, device=dev), torch.randn(rows, 2 * W, device=dev)
        for top in (2, 6):
            yp, wt, pos = torch.randn(rows * top, W, device=dev), torch.rand(rows * top, device=dev), torch.arange(rows * top, device=dev, dtype=torch.int32)
            moe = pkg.Moe(64, top, weight=P(wt), pos=P(pos))
            for two in (False, True):
                j = pkg.GatedJoin(P(a), P(b) if two else None, W, P(w) if two else None, P(w) if two else None, P(yp), W, C.pointer(moe), P(gates), P(gates, 4 * W), 2 * W)
                add(f"gated_join ({top} experts{', two mixers' if two else ''})", f"{rows}x{W}",
                    T.us([lambda s, x=x: ck(lib.cmlb200_gated_join_rows(j, P(x), P(w), 1e-5, rows, W, P(h), pkg.DT_BF16, W, s)) for x in xs], 4),
                    rows * W * (8.0 + 4 + 8 + 2 + 4 * top + (4 if two else 0)))
            add(f"  like: residual_add ({top} experts)", f"{rows}x{W}",
                T.us([lambda s, x=x: ck(lib.cmlb200_residual_add(P(x), P(yp), W, moe, P(w), 1e-5, rows, W, P(h), pkg.DT_BF16, W, s)) for x in xs], 4), rows * W * (8.0 + 2 + 4 * top))
        add("  like: residual_norm", f"{rows}x{W}", T.us([lambda s, x=x: ck(lib.cmlb200_residual_norm(P(x), P(a), W, P(w), P(w), 1e-5, rows, W, None, P(h), pkg.DT_BF16, W, s)) for x in xs], 4),
            rows * W * 14.0)
        del xs
        torch.cuda.empty_cache()


def plan(pkg, torch, E, top, rows):
    dev, align = torch.device("cuda:0"), 1 if rows <= 32 else 128
    n = pkg.lib.cmlb200_moe_positions(rows, top, E, align)
    i = lambda k: torch.zeros(k, device=dev, dtype=torch.int32)
    t = {"ids": i(rows * top), "weight": torch.zeros(rows * top, device=dev), "pos": i(rows * top), "src": i(n), "expert": i(n), "start": i(E), "count": i(E), "active": i(E), "num_active": i(1),
         "tiles": i(4 * (n // 128 + E + 1)), "num_tiles": i(1)}
    return t, pkg.Moe(E, top, **{k: P(v) for k, v in t.items()}), n, align


def routing(pkg, torch, T, add):
    dev, lib, ck, E, top = torch.device("cuda:0"), pkg.lib, pkg.check, 64, 6
    for rows in (1, 8, 32, 512, 2048):
        keep, like, _, align = plan(pkg, torch, E, top, rows)
        m = pkg.Moe.from_buffer_copy(like)
        m.sigmoid, m.group_best, m.groups, m.keep = 1, 2, 8, 4
        z = torch.randn(rows, E, device=dev)
        for name, a in (("moe_route (sigmoids, groups)", m), ("  like: moe_route", like)):
            add(name, f"{rows} rows, {top} of {E}", T.us([lambda s: ck(lib.cmlb200_moe_route(a, P(z), E, rows, align, s))], 32), rows * E * 4.0)


def experts(pkg, torch, T, add):
    """Up products without a gate beside gated ones of as many weights."""
    dev, lib, ck, E, top, W, ff = torch.device("cuda:0"), pkg.lib, pkg.check, 64, 6, 2048, 1408
    for rows in (1, 8, 32, 128, 512, 2048):
        keep, m, n, align = plan(pkg, torch, E, top, rows)
        z = torch.randn(rows, E, device=dev)
        ck(lib.cmlb200_moe_route(m, P(z), E, rows, align, None))
        torch.cuda.synchronize()
        used = int(keep["num_active"].item())
        x, f = torch.randn(rows if rows <= 32 else n, W, device=dev).bfloat16(), torch.empty(n, 2 * ff, device=dev, dtype=torch.bfloat16)
        wu, wg = torch.randn(E * ff, W, device=dev).bfloat16(), torch.randn(E * 2 * ff, W, device=dev).bfloat16()
        up, glu = pkg.Dense(pkg.DT_BF16, E * ff, W, W, P(wu)), pkg.Dense(pkg.DT_BF16, E * 2 * ff, W, W, P(wg))
        pairs = rows * top
        if rows <= 32:
            a = lambda s: ck(lib.cmlb200_moe_gemv_act(m, up, P(x), W, 1, rows, ff, pkg.ACT_GELU_ERF, P(f), 2 * ff, s))
            b = lambda s: ck(lib.cmlb200_moe_gemv_glu(m, glu, P(x), W, 1, rows, ff, pkg.ACT_GELU_TANH, 0.0, P(f), 2 * ff, s))
        else:
            a = lambda s: ck(lib.cmlb200_moe_gemm_act(m, up, P(x), W, rows, ff, pkg.ACT_GELU_ERF, P(f), 2 * ff, s))
            b = lambda s: ck(lib.cmlb200_moe_gemm_glu(m, glu, P(x), W, rows, ff, pkg.ACT_GELU_TANH, 0.0, P(f), 2 * ff, s))
        # between launches the caches are swept by another buffer's weights
        sweep = torch.empty(256 << 20, device=dev, dtype=torch.uint8)
        for name, g, k in (("moe_gemv_act" if rows <= 32 else "moe_gemm_act", a, 1), ("  like: moe_gemv_glu" if rows <= 32 else "  like: moe_gemm_glu", b, 2)):
            both = T.us([lambda s: (lib.cmlb200_memset(P(sweep), 0, len(sweep), s), g(s))], 4)
            alone = T.us([lambda s: lib.cmlb200_memset(P(sweep), 0, len(sweep), s)], 4)
            add(name, f"{rows} rows, {used} of {E} chosen", both - alone, 2.0 * used * k * ff * W + pairs * (2.0 * W + 2 * ff), 2.0 * pairs * k * ff * W)


def run(pkg, synth, torch, peaks, sampler, kernels_only=False, models_only=False):
    out = {"loops": True, "data": "synthetic", "dtype": "bf16", "unit": "tok/s", "peaks": peaks,
           "config": {"prompts": PROMPTS, "new_tokens": NEW, "l2": "weights, caches and states of a step are larger than L2; decode kernels rotate over copies, experts' products follow a sweep of L2"}}
    sampler.start()
    if not models_only:
        out["kernels"] = kernel_table(pkg, torch, peaks)
    if not kernels_only:
        sizes = lambda c: {k: v for k, v in c.items() if k != "batches"}
        out["4096"] = {"sizes": sizes(SIZES), "loops_bf16": leg(pkg, synth, torch, SIZES, peaks), "grouped_bf16": layered_leg(pkg, synth, torch, bench_latent.GROUPED, peaks)}
        torch.cuda.empty_cache()
        like = dict(bench_latent.EXPERTS)
        out["2048_experts"] = {"sizes": sizes(EXPERTS), "loops_bf16": leg(pkg, synth, torch, EXPERTS, peaks),
                               "latent_bf16": bench_latent.leg(pkg, synth, torch, bench_latent.mixed_config(synth, like), like, peaks)}
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
