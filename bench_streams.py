"""Throughput of models with residual streams, kept-window attention, chunked attention beside a gated delta rule, and experts
picked within groups (`python bench.py --streams`), beside the framework's closest models at equal layer sizes, and every
kernel against its roofline with the like kernel of those models under it. Random weights; layers (and experts) share bytes
on disk and are separate copies on the device. Not part of the default workload."""
import ctypes as C
import json

import numpy as np

import bench_latent
from bench_layered import NEW, PROMPTS, Timer, copies_for, layered_leg, model_leg

BATCHES = (1, 8, 32)
SIZES = dict(vocab=32000, width=4096, streams=4, heads=32, kv_heads=32, dim=128, left=(16, 4, 128, 128, 1024), right=(16, 16, 128, 128, 4), ranks=(128, 128), ff=11008, layers=8,
             window=1024, keep=4, batches=BATCHES)
EXPERTS = dict(SIZES, width=2048, heads=16, kv_heads=16, left=(8, 2, 128, 128, 1024), right=(8, 8, 128, 128, 4), ff=10944, experts=64, identity=16, groups=8, group_keep=4, top=6,
               expert_ff=1408, shared=2816)


def config(synth, c):
    """Attention and parallel layers in turn; experts in all but the first where there are any."""
    out = []
    for i in range(c["layers"]):
        mlp = synth.routed_mlp(c["experts"], c["identity"], c["top"], c["groups"], c["group_keep"], c["expert_ff"], c["shared"]) if i and "experts" in c else c["ff"]
        out.append(synth.parallel_layer(c["left"], c["right"], c["ranks"], mlp) if i % 2 else synth.kept_layer(c["heads"], c["kv_heads"], c["dim"], c["window"], c["keep"], mlp))
    return synth.streams_config(c["vocab"], c["width"], c["streams"], out, cap=15.0)


def leg(pkg, synth, torch, c, peaks):
    cfg, W = config(synth, c), c["width"]
    body, per_expert, moe, cache, state = 0, 0, 0, 0, 0
    for layer in cfg["layers"]:
        m, f = layer["mixer"], layer["mlp"]
        if layer["type"] == "attention":
            H, G, D = m["heads"], m["kv_heads"], m["dim"]
            body += W * D * (2 * H + G)
            cache += 4 * G * D
        else:
            a, r, ranks = m["left"], m["right"], layer["ranks"]
            body += W * (a["heads"] * (a["dim"] + a["vdim"]) + a["kv_heads"] * (a["dim"] + a["vdim"]))
            body += W * (2 * r["kv_heads"] * r["dim"] + 2 * r["heads"] * r["vdim"] + r["heads"] + sum(ranks)) + r["heads"] * (r["dim"] * ranks[0] + r["vdim"] * ranks[1])
            cache += 2 * a["kv_heads"] * (a["dim"] + a["vdim"])
            state += 8 * r["heads"] * r["dim"] * r["vdim"]
        if f["kind"] == "dense":
            body += 3 * W * f["ff"]
        else:
            moe += 1
            per_expert = 3 * W * f["expert"]["ff"]
            body += 3 * W * f["shared"]["ff"] + W * (f["router"]["experts"] + f["router"]["identity"])
    E, n, top = c.get("experts", 0), c.get("experts", 0) + c.get("identity", 0), c.get("top", 0)
    chosen = lambda B: E * (1 - (1 - top / n) ** B) if E else 0          # expected number of different experts of a step
    used = top * E / n if E else 0
    return model_leg(pkg, synth, torch, cfg, c, peaks, body + moe * per_expert * used, lambda B: body + moe * per_expert * chosen(B) + c["vocab"] * W, lambda: cache, state,
                     synth.streams_weight)


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

    attention(pkg, torch, T, add)
    delta(pkg, torch, T, add)
    joins(pkg, torch, T, add)
    routing(pkg, torch, T, add)
    products(pkg, torch, T, add)
    return out


def descriptor(pkg, torch, kind, H, G, D, k, v, table, per, keep, window=0, first=0):
    """kind: "kept" (values are keys, norms per head, distance bias), "chunk" (learned sink), or "like": the other layered design."""
    dev = k.device
    t = {"slopes": torch.rand(H, device=dev), "q": torch.ones(H * D, device=dev), "k": torch.ones(G * D, device=dev), "sinks": torch.randn(H, device=dev)}
    keep.append(t)
    pools = (pkg.DT_F16, k.data_ptr(), v.data_ptr(), 16, table.data_ptr(), per)
    if kind == "like":
        return pkg.Attn(H, G, D, D, D, D, D ** -0.5, window, t["slopes"].data_ptr(), 1, t["q"].data_ptr(), t["k"].data_ptr(), 1e-5, 0.1, 512.0, H * D + 2 * G * D, *pools)
    if kind == "kept":
        return pkg.Attn(H, G, D, D, D, D, D ** -0.5, window, t["slopes"].data_ptr(), 0, t["q"].data_ptr(), t["k"].data_ptr(), 1e-5, 0, 0, -1, *pools, 0, first, 0, None, 1, 1, 0)
    return pkg.Attn(H, G, D, D, D, D, D ** -0.5, 0, None, 1, None, None, 1e-5, 0, 0, -1, *pools, 0, 0, window, t["sinks"].data_ptr(), 0, 0, 0.8)


def attention(pkg, torch, T, add):
    dev, lib, ck, D = torch.device("cuda:0"), pkg.lib, pkg.check, 128
    # decoded tokens behind 1,024 and 8,192 tokens; a window of 1,024 with four kept ones, a chunk that has 1,024 tokens
    for B in BATCHES:
        for kind, H, G, ctx, window, first in (("kept", 32, 32, 1028, 0, 0), ("kept", 32, 32, 8191, 1024, 4), ("like", 32, 32, 1028, 0, 0), ("like", 32, 32, 8191, 1024, 0),
                                               ("chunk", 16, 4, 8191, 1024, 0), ("like", 16, 4, 8191, 1024, 0), ("chunk", 64, 8, 8191, 1024, 0), ("like", 64, 8, 8191, 1024, 0)):
            per, keep = ctx // 16 + 1, []
            seen = min(ctx, window + first) if window else ctx
            n = min(24, copies_for(4 * B * seen * G * D))
            blocks = B * per
            while n > 1 and n * blocks * 16 * G * D * 4 > 24e9:
                n -= 1
            table = torch.arange(blocks, device=dev, dtype=torch.int32).view(B, per).contiguous()
            pools = [(torch.randn(blocks * 16, G, D, device=dev, dtype=torch.float16), torch.randn(blocks * 16, G, D, device=dev, dtype=torch.float16)) for _ in range(n)]
            at = [descriptor(pkg, torch, kind, H, G, D, k, v, table, per, keep, window, first) for k, v in pools]
            ld = H * D + 2 * G * D + H
            qkv, o = torch.randn(B, ld, device=dev), torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
            pos, slot = torch.full((B,), ctx, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32)
            calls = [lambda s, a=a: ck(lib.cmlb200_attention_one(a, qkv.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), B, ctx, o.data_ptr(), H * D, s)) for a in at]
            name = "  like: attention_one" if kind == "like" else f"attention_one ({kind})"
            add(name, f"H={H} G={G} B={B} ctx={ctx} window={window}", T.us(calls, 8), 4.0 * B * seen * G * D, 4.0 * B * H * seen * D)
            del pools
            torch.cuda.empty_cache()
    for n in PROMPTS:
        for kind, H, G, window, first in (("kept", 32, 32, 0, 0), ("like", 32, 32, 0, 0), ("kept", 32, 32, 256, 4), ("like", 32, 32, 256, 0), ("chunk", 64, 8, 4096, 0), ("like", 64, 8, 0, 0),
                                          ("chunk", 64, 8, 256, 0)):
            per, keep = n // 16 + 1, []
            table = torch.arange(per, device=dev, dtype=torch.int32).view(1, per).contiguous()
            k, v = torch.randn(per * 16, G, D, device=dev).half(), torch.randn(per * 16, G, D, device=dev).half()
            a = descriptor(pkg, torch, kind, H, G, D, k, v, table, per, keep, window, first)
            ld = H * D + 2 * G * D + H
            qkv, o = torch.randn(n, ld, device=dev), torch.empty(n, H * D, device=dev, dtype=torch.bfloat16)
            tiles = torch.tensor([[i, 64, 0, i] for i in range(0, n, 64)], device=dev, dtype=torch.int32)
            pos, slot = torch.arange(n, device=dev, dtype=torch.int32), torch.zeros(n, device=dev, dtype=torch.int32)
            p = np.arange(n)
            pairs = float((p - p // window * window + 1).sum()) if kind == "chunk" else float(np.minimum(p + 1, (window or n) + first).sum())
            name = "  like: " if kind == "like" else ""
            add(f"{name}attention_tiles" + ("" if name else f" ({kind})"), f"H={H} G={G} rows={n} window={window}",
                T.us([lambda s: ck(lib.cmlb200_attention_tiles(a, qkv.data_ptr(), ld, tiles.data_ptr(), len(tiles), o.data_ptr(), H * D, s))], 10), 0, 4.0 * pairs * H * D)
            if window == 0:
                cols = H * D + (1 if kind == "kept" else 2) * G * D
                add(f"{name}qk_norm_append" + ("" if name else f" ({kind})"), f"H={H} G={G} rows={n}",
                    T.us([lambda s: ck(lib.cmlb200_qk_norm_append(a, qkv.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), n, s))], 10), n * (4.0 * cols + 4 * H * D + 4 * G * D))


def delta(pkg, torch, T, add):
    dev, lib, ck, D, taps = torch.device("cuda:0"), pkg.lib, pkg.check, 128, 4
    P = lambda t: t.data_ptr()

    def layer(H, G, slots):
        ch = 2 * G * D + H * D
        k = [torch.randn(taps, ch, device=dev) / 2, torch.rand(H, device=dev) * 0.1, torch.randn(H * D, device=dev), torch.ones(D, device=dev), torch.randn(slots, H, D, D, device=dev),
             torch.randn(slots, taps, ch, device=dev)]
        return pkg.Delta(H, G, D, D, taps, D, 0, P(k[0]), P(k[1]), P(k[2]), P(k[3]), 1e-5, 0.0, P(k[4]), P(k[5])), k, ch
    for H, G in ((16, 16), (32, 32), (32, 8)):
        for B in BATCHES:
            n = min(64, copies_for(8 * B * H * D * D))
            ls = [layer(H, G, B) for _ in range(n)]
            ch = ls[0][2]
            ld = ch + H
            proj, dec, gate = torch.randn(B, ld, device=dev), torch.randn(B, H * D, device=dev), torch.randn(B, H * D, device=dev)
            pos, slot, o = torch.full((B,), 99, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32), torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
            calls = [lambda s, a=l[0]: ck(lib.cmlb200_delta_one(a, P(proj), ld, P(dec), H * D, P(gate), H * D, P(pos), P(slot), B, P(o), pkg.DT_BF16, H * D, s)) for l in ls]
            add("delta_one", f"H={H} G={G} B={B}", T.us(calls, 8), B * (8.0 * H * D * D + 4.0 * (taps + 1) * ch + 10 * H * D), flops32=8.0 * B * H * D * D)
            del ls
            torch.cuda.empty_cache()
        for seqs, n in ((1, 64), (1, 512), (1, 2048), (4, 512)):
            a, keep, ch = layer(H, G, seqs)
            rows, ld = seqs * n, ch + H
            proj, dec0, gate = torch.randn(rows, ld, device=dev), torch.randn(rows, H * D, device=dev), torch.randn(rows, H * D, device=dev)
            pos, slot = torch.arange(n, device=dev, dtype=torch.int32).repeat(seqs), torch.arange(seqs, device=dev, dtype=torch.int32).repeat_interleave(n)
            runs = torch.tensor([[i * n, n, i, 0] for i in range(seqs)], device=dev, dtype=torch.int32)
            w, o = torch.empty(lib.cmlb200_delta_work_floats(a, rows, seqs), device=dev), torch.empty(rows, H * D, device=dev, dtype=torch.bfloat16)
            us = T.us([lambda s: ck(lib.cmlb200_delta_rows(a, P(proj), ld, P(dec0), H * D, P(gate), H * D, P(pos), P(slot), 0, rows, P(runs), seqs, P(w), P(o), pkg.DT_BF16, H * D, s))], 10)
            # bytes: projections, decays and gates in, outputs out, the state once. Operations: decay, two sums, one update per element of the state
            add("delta_rows (3 launches)", f"H={H} G={G} {seqs} x {n} rows", us, rows * (4.0 * ch + 8.0 * H * D + 2 * H * D) + 8.0 * seqs * H * D * D, flops32=7.0 * rows * H * D * D)


def joins(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    P = lambda t: t.data_ptr()
    for S in (2, 4):
        for rows, dim in ((1, 4096), (8, 4096), (32, 4096), (512, 4096), (2048, 4096)):
            n = min(copies_for(rows * dim * (8 * S + 6)), 64)
            xs = [torch.randn(rows, S, dim, device=dev) for _ in range(n)]
            y, h, w = torch.randn(rows, dim, device=dev), torch.empty(rows, dim, device=dev, dtype=torch.bfloat16), torch.ones(dim, device=dev)
            c = [torch.eye(S, device=dev), torch.ones(S, device=dev), torch.ones(S, device=dev)]
            hc = pkg.Streams(S, P(c[0]), P(c[1]), P(c[2]))
            add(f"stream_join ({S} streams)", f"{rows}x{dim}", T.us([lambda s, x=x: ck(lib.cmlb200_stream_join(hc, P(x), P(y), dim, None, P(w), 1e-5, rows, dim, None, P(h), pkg.DT_BF16, dim, s))
                                                                  for x in xs], 4), rows * dim * (8.0 * S + 6))
            yp, add_rows, wt, sw = torch.randn(rows * 6, dim, device=dev), torch.randn(rows, dim, device=dev), torch.rand(rows * 6, device=dev), torch.rand(rows, device=dev)
            pos = torch.arange(rows * 6, device=dev, dtype=torch.int32)
            pos[::6] = -1                              # one identity expert a row
            moe = pkg.Moe(64, 6, weight=P(wt), pos=P(pos), identity=16, self=P(sw))
            j = pkg.Join(C.pointer(moe), P(h), P(add_rows), dim)
            add(f"stream_join ({S} streams, 5 experts, identity, shared)", f"{rows}x{dim}",
                T.us([lambda s, x=x: ck(lib.cmlb200_stream_join(hc, P(x), P(yp), dim, j, P(w), 1e-5, rows, dim, None, P(h), pkg.DT_BF16, dim, s)) for x in xs], 4),
                rows * dim * (8.0 * S + 2 + 20 + 2 + 4))
            if S == 2:
                x1 = [torch.randn(rows, dim, device=dev) for _ in range(min(copies_for(rows * dim * 14), 64))]
                add("  like: residual_norm", f"{rows}x{dim}", T.us([lambda s, x=x: ck(lib.cmlb200_residual_norm(P(x), P(y), dim, P(w), P(w), 1e-5, rows, dim, None, P(h), pkg.DT_BF16, dim, s))
                                                                   for x in x1], 4), rows * dim * 14.0)
                del x1
            del xs
            torch.cuda.empty_cache()
    for rows, dim in ((1, 4096), (2048, 4096)):
        table, tok = torch.randn(32000, dim, device=dev).bfloat16(), torch.randint(0, 32000, (rows,), device=dev, dtype=torch.int32)
        x, pos = torch.empty(rows, 4, dim, device=dev), torch.zeros(rows, device=dev, dtype=torch.int32)
        add("embed_streams (4 streams)", f"{rows}x{dim}", T.us([lambda s: ck(lib.cmlb200_embed_streams(P(table), pkg.DT_BF16, P(tok), 2.0, 4, rows, dim, 32000, P(x), s))], 10), rows * dim * 18.0)
        add("  like: embed_rows", f"{rows}x{dim}", T.us([lambda s: ck(lib.cmlb200_embed_rows(P(table), pkg.DT_BF16, P(tok), P(pos), None, rows, dim, 32000, P(x), s))], 10), rows * dim * 6.0)


def routing(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    E, I, top = 64, 16, 6
    i = lambda k: torch.zeros(k, device=dev, dtype=torch.int32)
    for rows in (1, 8, 32, 512, 2048):
        align = 1 if rows <= 32 else 128
        n = lib.cmlb200_moe_positions(rows, top, E + I, align)
        t = {"ids": i(rows * top), "weight": torch.zeros(rows * top, device=dev), "pos": i(rows * top), "src": i(n), "expert": i(n), "start": i(E + I), "count": i(E + I), "active": i(E + I),
             "num_active": i(1), "tiles": i(4 * (n // 128 + E + I + 1)), "num_tiles": i(1), "self": torch.zeros(rows, device=dev)}
        p = {k: v.data_ptr() for k, v in t.items()}
        z, corr = torch.randn(rows, E + I, device=dev), torch.randn(E + I, device=dev)
        m, like = pkg.Moe(E, top, identity=I, groups=8, keep=4, correction=corr.data_ptr(), normalize=1, scale=1.5, **p), pkg.Moe(E + I, top, **{k: v for k, v in p.items() if k != "self"})
        for name, a in (("moe_route (groups)", m), ("  like: moe_route", like)):
            add(name, f"{rows} rows, {top} of {E + I}", T.us([lambda s: ck(lib.cmlb200_moe_route(a, z.data_ptr(), E + I, rows, align, s))], 32), rows * (E + I) * 4.0)


def products(pkg, torch, T, add):
    """The second factors of decays and gates, a projection with a bias, the vocabulary projection with a cap."""
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    P = lambda t: t.data_ptr()
    for N, K, bias, cap, what in ((2048, 128, False, 0.0, "second factor"), (12288, 4096, True, 0.0, "bias"), (12288, 4096, False, 0.0, "like: no bias"), (32000, 4096, False, 15.0, "cap"),
                                  (32000, 4096, False, 0.0, "like: no cap")):
        n = copies_for(N * K * 2)
        ws, b = [torch.randn(N, K, device=dev).bfloat16() for _ in range(n)], torch.randn(N, device=dev)
        W = [pkg.Dense(pkg.DT_BF16, N, K, K, P(w), P(b) if bias else None, cap) for w in ws]
        for M in (1, 8, 32, 512, 2048):
            if M > 256 and N == 32000:
                continue
            x, y = torch.randn(M, K, device=dev).bfloat16(), torch.empty(M, N, device=dev)
            f = lib.cmlb200_gemv_dense if M <= 32 else lib.cmlb200_gemm_dense
            add(f"{'gemv' if M <= 32 else 'gemm'}_dense ({what})", f"{N}x{K} M={M}", T.us([lambda s, w=w: ck(f(w, P(x), K, M, P(y), N, s)) for w in W], 4), N * K * 2.0 + M * (K * 2.0 + N * 4),
                2.0 * M * N * K)
        del ws
        torch.cuda.empty_cache()
    for rows in (1, 32, 2048):
        x, o = torch.randn(rows, 10512, device=dev), torch.empty(rows, 256, device=dev, dtype=torch.bfloat16)
        add("pack_columns", f"{rows}x256", T.us([lambda s: ck(lib.cmlb200_pack_columns(P(x), 10512, 9232, 128, 128, 128, rows, P(o), 256, s))], 10), rows * 256 * 6.0)


def run(pkg, synth, torch, peaks, sampler, kernels_only=False, models_only=False):
    out = {"streams": True, "data": "synthetic", "dtype": "bf16", "unit": "tok/s", "peaks": peaks,
           "config": {"prompts": PROMPTS, "new_tokens": NEW, "l2": "weights, caches and states of a step are larger than L2; decode kernels rotate over copies"}}
    sampler.start()
    if not models_only:
        out["kernels"] = kernel_table(pkg, torch, peaks)
    if not kernels_only:
        sizes = lambda c: {k: v for k, v in c.items() if k != "batches"}
        out["4096_dense"] = {"sizes": sizes(SIZES), "streams_bf16": leg(pkg, synth, torch, SIZES, peaks), "grouped_bf16": layered_leg(pkg, synth, torch, bench_latent.GROUPED, peaks)}
        torch.cuda.empty_cache()
        like = dict(bench_latent.EXPERTS)
        out["2048_experts"] = {"sizes": sizes(EXPERTS), "streams_bf16": leg(pkg, synth, torch, EXPERTS, peaks),
                               "latent_bf16": bench_latent.leg(pkg, synth, torch, bench_latent.mixed_config(synth, like), like, peaks)}
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
