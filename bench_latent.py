"""Throughput of models with latent attention, polynomial feed-forwards and experts (`python bench.py --latent`) beside the
layered model with grouped heads at equal layer sizes, and every kernel against its roofline with the like kernel of that
model under it. Random weights; layers (and experts) share bytes on disk and are separate copies on the device. Not part of
the default workload."""
import ctypes as C
import json

import numpy as np

from bench_layered import NEW, PROMPTS, Timer, copies_for, layered_leg, model_leg

BATCHES = (1, 8, 32)
# equal width, heads, head sizes and feed-forward
GROUPED = dict(vocab=32000, width=4096, heads=32, kv_heads=32, dim=128, ff=11008, layers=8, window=1024, batches=BATCHES)
SIZES = dict(vocab=32000, width=4096, heads=32, dim=128, rot=64, vdim=128, rank=512, ff=11008, layers=8, window=1024, batches=BATCHES)
EXPERTS = dict(SIZES, width=2048, heads=16, ff=10944, experts=64, top=6, expert_ff=1408)


def dense_config(synth, c):
    layer = lambda: synth.latent_layer(c["heads"], c["dim"], c["rot"], c["vdim"], c["rank"], c["ff"])
    return synth.latent_config(c["vocab"], c["width"], [layer() for _ in range(c["layers"])])


def mixed_config(synth, c):
    """Full and windowed gated layers in turn, every fourth layer on an earlier one's cache, experts in all but the first."""
    out = []
    for i in range(c["layers"]):
        mlp = (c["experts"], c["top"], c["expert_ff"], 7.0) if i else c["ff"]
        gated = i % 2 == 1
        out.append(synth.latent_layer(c["heads"], c["dim"], c["rot"], c["vdim"], c["rank"], mlp, c["window"] if gated else None, gated,
                                      scaling=(8.0, 4096, 32.0, 1.0) if gated else None, kv_from=i - 2 if i % 4 == 2 else None))
    return synth.latent_config(c["vocab"], c["width"], out)


def leg(pkg, synth, torch, cfg, c, peaks):
    W, attn, dense, per_expert, moe, own = c["width"], 0, 0, 0, 0, 0
    for layer in cfg["layers"]:
        m, f = layer["mixer"], layer["mlp"]
        H, R = m["heads"], m["kv_rank"]
        attn += W * H * (m["dim"] + m["rot_dim"]) + H * (m["dim"] + m["vdim"]) * R + W * H * m["vdim"] + (W * H * m["vdim"] if layer["type"].endswith("_2") else 0)
        attn += W * (R + m["rot_dim"]) if m.get("kv_from") is None else 0
        if f["kind"] == "dense":
            dense += 2 * W * f["ff"]
        else:
            moe += 1
            per_expert = 3 * W * f["expert"]["ff"]
            attn += W * f["router"]["experts"]
    E, top = c.get("experts", 0), c.get("top", 0)
    chosen = lambda B: E * (1 - (1 - top / E) ** B) if E else 0          # expected number of different experts of a step
    weights = lambda B: attn + dense + moe * per_expert * chosen(B) + c["vocab"] * W
    cache = 2 * len(cfg["layers"]) * (c["rank"] + c["rot"])
    return model_leg(pkg, synth, torch, cfg, c, peaks, attn + dense + moe * per_expert * top, weights, lambda: cache)


# ---- kernels -------------------------------------------------------------------------------------------------
def kernel_table(pkg, synth, torch, peaks):
    dev, lib, ck, T, out = torch.device("cuda:0"), pkg.lib, pkg.check, Timer(torch), []

    def add(kernel, shape, us, nbytes=0.0, flops=0.0):
        """The roofline of a launch is the slower of its bytes and its operations."""
        tb, tf = nbytes / peaks["hbm_gbs"] / 1e3, flops / peaks["bf16_tflops"] / 1e6
        out.append({"kernel": kernel, "shape": shape, "us": round(us, 2), "bound": "tensor" if tf > tb else "hbm", "frac": round(max(tb, tf) / us, 4)})

    heads_rows(pkg, torch, T, add)
    attention(pkg, torch, T, add)
    rows_and_norms(pkg, torch, T, add)
    experts(pkg, torch, T, add)
    return out


def latent(pkg, torch, H, B, ctx, rows_of_table=None, D=128, P=64, V=128, R=512, proj_extra=0):
    """A layer's descriptor, its tensors, and the pool's number of blocks."""
    dev = torch.device("cuda:0")
    per = (ctx + 15) // 16 + 1
    keep = {"norm": torch.ones(R, device=dev), "freq": torch.rand(P // 2, device=dev), "table": torch.arange(B * per, device=dev, dtype=torch.int32).view(B, per).contiguous()}
    ld, q = (R + P + 15) // 16 * 16, H * (D + P)
    keep["pool"] = torch.randn(B * per * 16, ld, device=dev).half()
    a = pkg.Latent(H, D, P, V, R, ld, (R + 63) // 64 * 64, (D + P) ** -0.5, 0, keep["norm"].data_ptr(), 1e-5, keep["freq"].data_ptr(), 1.0, q, -1, pkg.DT_F16,
                   keep["pool"].data_ptr(), 16, keep["table"].data_ptr(), per, B * per)
    return a, keep, q + R + P


def heads_rows(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    for H in (32, 128):
        a, keep, ld = latent(pkg, torch, H, 32, 64)
        n = copies_for(H * 512 * 128 * 2)
        w = [torch.randn(H, 512, 128, device=dev).bfloat16() for _ in range(n)]
        wv = [torch.randn(H, 128, 512, device=dev).bfloat16() for _ in range(n)]
        for M in (1, 8, 32):
            proj, pos, slot = torch.randn(M, ld, device=dev), torch.full((M,), 5, device=dev, dtype=torch.int32), torch.arange(M, device=dev, dtype=torch.int32)
            q, o, y = torch.zeros(M, H, a.ld, device=dev).half(), torch.randn(M, H, 512, device=dev).bfloat16(), torch.zeros(M, H * 128, device=dev).bfloat16()
            calls = [lambda s, t=t: ck(lib.cmlb200_latent_query(a, t.data_ptr(), proj.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), M, q.data_ptr(), s)) for t in w]
            add("latent_query", f"H={H} M={M}", T.us(calls, 4), H * 512 * 128 * 2 + M * H * (192 * 4 + 576 * 2))
            calls = [lambda s, t=t: ck(lib.cmlb200_latent_output(a, t.data_ptr(), o.data_ptr(), proj.data_ptr(), ld, M, y.data_ptr(), H * 128, s)) for t in wv]
            add("latent_output", f"H={H} M={M}", T.us(calls, 4), H * 512 * 128 * 2 + M * H * (512 * 2 + 128 * 2))
            if H == 32:
                ws = [torch.randn(4096, 512, device=dev).bfloat16() for _ in range(n)]
                W = [pkg.Dense(pkg.DT_BF16, 4096, 512, 512, t.data_ptr()) for t in ws]
                x, yy = torch.randn(M, 512, device=dev).bfloat16(), torch.empty(M, 4096, device=dev)
                add("  like: gemv_dense", f"4096x512 M={M}", T.us([lambda s, d=d: ck(lib.cmlb200_gemv_dense(d, x.data_ptr(), 512, M, yy.data_ptr(), 4096, s)) for d in W], 4),
                    4096 * 512 * 2 + M * (512 * 2 + 4096 * 4))
        del w, wv
        torch.cuda.empty_cache()


def grouped(pkg, torch, H, G, D, k, v, table, per, keep):
    slopes, qn, kn = torch.rand(H, device=k.device), torch.ones(H * D, device=k.device), torch.ones(G * D, device=k.device)
    keep += [slopes, qn, kn]
    return pkg.Attn(H, G, D, D, D, D, D ** -0.5, 0, slopes.data_ptr(), 1, qn.data_ptr(), kn.data_ptr(), 1e-5, 0.1, 512.0, H * D + 2 * G * D, pkg.DT_F16, k.data_ptr(), v.data_ptr(),
                    16, table.data_ptr(), per)


def attention(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    D, P, V, R = 128, 64, 128, 512
    i32 = lambda *a: torch.tensor(a, device=dev, dtype=torch.int32)
    # decoded tokens
    for ctx in (1024, 8192):
        for B in BATCHES:
            for H in (32, 128):
                n = min(24, copies_for(B * ctx * (R + P) * 2))
                ls = [latent(pkg, torch, H, B, ctx) for _ in range(n)]
                q, o = torch.randn(B, H, ls[0][0].ld, device=dev).half(), torch.zeros(B, H, R, device=dev).bfloat16()
                pos, slot = torch.full((B,), ctx, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32)
                calls = [lambda s, a=l[0]: ck(lib.cmlb200_attention_latent(a, q.data_ptr(), B, pos.data_ptr(), slot.data_ptr(), B, ctx, None, 0, o.data_ptr(), s)) for l in ls]
                add("attention_latent", f"H={H} B={B} ctx={ctx}", T.us(calls, 8), 2.0 * B * ctx * (R + P) + 2.0 * B * H * (2 * R + P), 2.0 * B * H * ctx * (2 * R + P))
                del ls
                torch.cuda.empty_cache()
            for H, G in ((32, 32), (64, 8)) if ctx == 1024 else ((64, 8),):
                per, keep = ctx // 16 + 1, []
                n = min(24, copies_for(4 * B * ctx * G * D))
                table = torch.arange(B * per, device=dev, dtype=torch.int32).view(B, per).contiguous()
                pools = [(torch.randn(B * per * 16, G, D, device=dev).half(), torch.randn(B * per * 16, G, D, device=dev).half()) for _ in range(n)]
                at = [grouped(pkg, torch, H, G, D, k, v, table, per, keep) for k, v in pools]
                ld = H * D + 2 * G * D + H
                qkv, o = torch.randn(B, ld, device=dev), torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
                calls = [lambda s, a=a: ck(lib.cmlb200_attention_one(a, qkv.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), B, ctx, o.data_ptr(), H * D, s)) for a in at]
                add("  like: attention_one", f"H={H} G={G} B={B} ctx={ctx}", T.us(calls, 8), 4.0 * B * ctx * G * D, 4.0 * B * H * ctx * D)
                del pools
                torch.cuda.empty_cache()
    # prompts
    for H in (32,):
        for n in PROMPTS:
            per = n // 16
            a, keep, ld = latent(pkg, torch, H, 1, n)
            proj, o = torch.randn(n, ld, device=dev), torch.empty(n, H * V, device=dev, dtype=torch.bfloat16)
            pos, slot = torch.arange(n, device=dev, dtype=torch.int32), torch.zeros(n, device=dev, dtype=torch.int32)
            tiles = torch.tensor([[i, 64, 0, i] for i in range(0, n, 64)], device=dev, dtype=torch.int32)
            k, v, c = torch.zeros(n, H, D + P, device=dev).half(), torch.zeros(n, H, V, device=dev).half(), torch.randn(n, R, device=dev).bfloat16()
            k.normal_(), v.normal_()
            tab = torch.arange(per + 1, device=dev, dtype=torch.int32).view(1, -1).contiguous()
            s2 = pkg.Attn(H, H, D + P, V, D + P, V, (D + P) ** -0.5, 0, None, 0, None, None, 0, 0, 0, -1, pkg.DT_F16, k.data_ptr(), v.data_ptr(), 16, tab.data_ptr(), a.table_ld, 0)
            pairs = n * (n + 1) / 2
            add("attention_tiles (expanded)", f"H={H} rows={n}",
                T.us([lambda s: ck(lib.cmlb200_attention_tiles(s2, proj.data_ptr(), ld, tiles.data_ptr(), len(tiles), o.data_ptr(), H * V, s))], 10), n * H * (192 * 4 + 256.0),
                2.0 * pairs * H * (D + P + V))
            kk, vv, kp = torch.randn(n, H, D, device=dev).half(), torch.randn(n, H, D, device=dev).half(), []
            g = grouped(pkg, torch, H, H, D, kk, vv, tab, a.table_ld, kp)
            lg = 3 * H * D + H
            qkv = torch.randn(n, lg, device=dev)
            add("  like: attention_tiles", f"H={H} G={H} rows={n}",
                T.us([lambda s: ck(lib.cmlb200_attention_tiles(g, qkv.data_ptr(), lg, tiles.data_ptr(), len(tiles), o.data_ptr(), H * D, s))], 10), 0, 4.0 * pairs * H * D)
            W = torch.randn(H * (D + V), R, device=dev).bfloat16()
            dW = pkg.Dense(pkg.DT_BF16, H * (D + V), R, R, W.data_ptr())
            add("latent_expand", f"H={H} keys={n}", T.us([lambda s: ck(lib.cmlb200_latent_expand(a, dW, c.data_ptr(), n, s2, s))], 10),
                2.0 * H * (D + V) * R + n * (R * 2.0 + H * (D + V) * 2), 2.0 * n * R * H * (D + V))
            y = torch.empty(n, H * (D + V), device=dev)
            add("  like: gemm_dense", f"{H * (D + V)}x{R} M={n}", T.us([lambda s: ck(lib.cmlb200_gemm_dense(dW, c.data_ptr(), R, n, y.data_ptr(), H * (D + V), s))], 10),
                2.0 * H * (D + V) * R + n * (R * 2.0 + H * (D + V) * 4), 2.0 * n * R * H * (D + V))
            keys = np.array([[0, 0, n, 0]], np.int32)
            add("latent_gather", f"H={H} keys={n}", T.us([lambda s: ck(lib.cmlb200_latent_gather(a, keys.ctypes.data, 1, c.data_ptr(), s2, s))], 10),
                n * ((R + P) * 2.0 + R * 2 + H * P * 2))
            add("latent_append", f"H={H} rows={n}", T.us([lambda s: ck(lib.cmlb200_latent_append(a, proj.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), n, s))], 10),
                n * (H * P * 8.0 + (R + P) * 6))
            add("  like: qk_norm_append", f"H={H} G={H} rows={n}",
                T.us([lambda s: ck(lib.cmlb200_qk_norm_append(g, qkv.data_ptr(), lg, pos.data_ptr(), slot.data_ptr(), n, s))], 10), n * (H * D * 8.0 + H * D * 8 + 4 * H * D))
        # a short portion behind a long history: over the latents, and what the grouped heads do
        for rows, ctx in ((16, 4096), (64, 1024), (64, 4096)):
            a, keep, ld = latent(pkg, torch, H, 1, ctx + rows)
            q, o = torch.randn(rows, H, a.ld, device=dev).half(), torch.zeros(rows, H, R, device=dev).bfloat16()
            tile = i32([0, rows, 0, ctx])
            pairs = rows * ctx + rows * (rows + 1) / 2
            add("attention_latent (portion)", f"H={H} rows={rows} ctx={ctx}",
                T.us([lambda s: ck(lib.cmlb200_attention_latent(a, q.data_ptr(), rows, None, None, 0, ctx + rows, tile.data_ptr(), 1, o.data_ptr(), s))], 10), 2.0 * ctx * (R + P), 2.0 * pairs * H * (2 * R + P))
            per, kp = (ctx + rows) // 16 + 1, []
            tab = torch.arange(per, device=dev, dtype=torch.int32).view(1, -1).contiguous()
            kk, vv = torch.randn(per * 16, H, D, device=dev).half(), torch.randn(per * 16, H, D, device=dev).half()
            g = grouped(pkg, torch, H, H, D, kk, vv, tab, per, kp)
            lg = 3 * H * D + H
            qkv, oo = torch.randn(rows, lg, device=dev), torch.empty(rows, H * D, device=dev, dtype=torch.bfloat16)
            add("  like: attention_tiles", f"H={H} G={H} rows={rows} ctx={ctx}",
                T.us([lambda s: ck(lib.cmlb200_attention_tiles(g, qkv.data_ptr(), lg, tile.data_ptr(), 1, oo.data_ptr(), H * D, s))], 10), 4.0 * ctx * H * D, 4.0 * pairs * H * D)


def rows_and_norms(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    for rows, dim in ((1, 4096), (8, 4096), (512, 4096), (2048, 4096)):
        n = min(copies_for(rows * dim * 14), 64)
        xs = [torch.randn(rows, dim, device=dev) for _ in range(n)]
        y, h, w = torch.randn(rows, dim, device=dev), torch.empty(rows, dim, device=dev, dtype=torch.bfloat16), torch.ones(dim, device=dev)
        add("residual_add", f"{rows}x{dim}", T.us([lambda s, x=x: ck(lib.cmlb200_residual_add(x.data_ptr(), y.data_ptr(), dim, None, w.data_ptr(), 1e-5, rows, dim, h.data_ptr(),
                                                                                           pkg.DT_BF16, dim, s)) for x in xs], 4), rows * dim * 14.0)
        yp = torch.randn(rows * 6, dim, device=dev)
        wt, pos = torch.rand(rows * 6, device=dev), torch.arange(rows * 6, device=dev, dtype=torch.int32)
        moe = pkg.Moe(64, 6, None, wt.data_ptr(), pos.data_ptr())
        add("residual_add (6 experts)", f"{rows}x{dim}", T.us([lambda s, x=x: ck(lib.cmlb200_residual_add(x.data_ptr(), yp.data_ptr(), dim, moe, w.data_ptr(), 1e-5, rows, dim,
                                                                                                       h.data_ptr(), pkg.DT_BF16, dim, s)) for x in xs], 4), rows * dim * 34.0)
        add("  like: residual_norm", f"{rows}x{dim}", T.us([lambda s, x=x: ck(lib.cmlb200_residual_norm(x.data_ptr(), y.data_ptr(), dim, w.data_ptr(), w.data_ptr(), 1e-5, rows, dim,
                                                                                                    None, h.data_ptr(), pkg.DT_BF16, dim, s)) for x in xs], 4), rows * dim * 14.0)
        del xs
        ff, coef = 11008, torch.ones(4, device=dev)
        n = min(copies_for(rows * ff * 6), 64)
        zs, f = [torch.randn(rows, ff, device=dev) for _ in range(n)], torch.empty(rows, ff, device=dev, dtype=torch.bfloat16)
        add("poly_norm", f"{rows}x{ff}", T.us([lambda s, z=z: ck(lib.cmlb200_poly_norm(z.data_ptr(), ff, rows, ff, coef.data_ptr(), 1e-5, f.data_ptr(), pkg.DT_BF16, ff, s)) for z in zs], 4),
            rows * ff * 6.0)
        del zs
        torch.cuda.empty_cache()


def experts(pkg, torch, T, add):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    E, top, ff, W = 64, 6, 1408, 2048
    n = 3
    gu, dn = [torch.randn(E * 2 * ff, W, device=dev).bfloat16() for _ in range(n)], [torch.randn(E * W, ff, device=dev).bfloat16() for _ in range(n)]
    G, Dn = [pkg.Dense(pkg.DT_BF16, E * 2 * ff, W, W, t.data_ptr()) for t in gu], [pkg.Dense(pkg.DT_BF16, E * W, ff, ff, t.data_ptr()) for t in dn]
    one_gu, one_dn = [pkg.Dense(pkg.DT_BF16, 2 * ff * top, W, W, t.data_ptr()) for t in gu], [pkg.Dense(pkg.DT_BF16, W * top, ff, ff, t.data_ptr()) for t in dn]
    i = lambda k: torch.zeros(k, device=dev, dtype=torch.int32)
    for rows in (1, 8, 32, 128, 512, 2048):
        align = 1 if rows <= 32 else 128
        P = lib.cmlb200_moe_positions(rows, top, E, align)
        t = {"ids": i(rows * top), "weight": torch.zeros(rows * top, device=dev), "pos": i(rows * top), "src": i(P), "expert": i(P), "start": i(E), "count": i(E), "active": i(E),
             "num_active": i(1), "tiles": i(4 * (P // 128 + E + 1)), "num_tiles": i(1)}
        m = pkg.Moe(E, top, **{k: v.data_ptr() for k, v in t.items()})
        z, x = torch.randn(rows, E, device=dev), torch.randn(rows, W, device=dev).bfloat16()
        xp, f, y = torch.randn(P, W, device=dev).bfloat16(), torch.randn(P, ff, device=dev).bfloat16(), torch.empty(P, W, device=dev)
        add("moe_route", f"{rows} rows, {top} of {E}", T.us([lambda s: ck(lib.cmlb200_moe_route(m, z.data_ptr(), E, rows, align, s))], 32), rows * E * 4.0)
        used = int(t["num_active"].item())
        if rows <= 32:
            add("moe_gemv_glu", f"{ff}x{W} rows={rows} ({used} experts)",
                T.us([lambda s, w=w: ck(lib.cmlb200_moe_gemv_glu(m, w, x.data_ptr(), W, 1, rows, ff, pkg.ACT_CLAMPED, 7.0, f.data_ptr(), ff, s)) for w in G], 8),
                used * 2.0 * 2 * ff * W)
            add("moe_gemv", f"{W}x{ff} rows={rows} ({used} experts)", T.us([lambda s, w=w: ck(lib.cmlb200_moe_gemv(m, w, f.data_ptr(), ff, 0, rows, W, y.data_ptr(), W, s)) for w in Dn], 8),
                used * 2.0 * ff * W)
            if rows == 1:
                ff6 = torch.empty(1, ff * top, device=dev).bfloat16()
                y6 = torch.empty(1, W * top, device=dev)
                add("  like: gemv_dense_glu", f"{ff * top}x{W} M=1", T.us([lambda s, w=w: ck(lib.cmlb200_gemv_dense_glu(w, x.data_ptr(), W, 1, ff * top, 1, ff6.data_ptr(), ff * top, s))
                                                                         for w in one_gu], 8), 4.0 * top * ff * W)
                add("  like: gemv_dense", f"{W * top}x{ff} M=1", T.us([lambda s, w=w: ck(lib.cmlb200_gemv_dense(w, f.data_ptr(), ff, 1, y6.data_ptr(), W * top, s)) for w in one_dn], 8),
                    2.0 * top * ff * W)
            continue
        add("moe_gather", f"rows={rows}", T.us([lambda s: ck(lib.cmlb200_moe_gather(m, x.data_ptr(), W, rows, W, xp.data_ptr(), W, s))], 8), rows * W * 2.0 * (1 + top))
        add("moe_gemm_glu", f"{ff}x{W} rows={rows} ({used} experts)",
            T.us([lambda s, w=w: ck(lib.cmlb200_moe_gemm_glu(m, w, xp.data_ptr(), W, rows, ff, pkg.ACT_CLAMPED, 7.0, f.data_ptr(), ff, s)) for w in G], 4),
            used * 4.0 * ff * W + rows * top * (W + ff) * 2.0, 4.0 * rows * top * ff * W)
        add("moe_gemm", f"{W}x{ff} rows={rows} ({used} experts)", T.us([lambda s, w=w: ck(lib.cmlb200_moe_gemm(m, w, f.data_ptr(), ff, rows, W, y.data_ptr(), W, s)) for w in Dn], 4),
            used * 2.0 * ff * W + rows * top * (ff * 2.0 + W * 4), 2.0 * rows * top * ff * W)
        # the same products with the rows' experts side by side: equal operations and weight bytes per row tile
        per = max(128, rows * top // E)
        xd, yd = torch.randn(per, W, device=dev).bfloat16(), torch.empty(per, E * ff, device=dev).bfloat16()
        yw, fd = torch.empty(per, E * W, device=dev), torch.randn(per, ff, device=dev).bfloat16()
        add("  like: gemm_dense_glu", f"{E * ff}x{W} M={per}", T.us([lambda s, w=w: ck(lib.cmlb200_gemm_dense_glu(w, xd.data_ptr(), W, per, E * ff, 1, yd.data_ptr(), E * ff, s)) for w in G], 4),
            4.0 * E * ff * W + per * (W + E * ff) * 2.0, 4.0 * per * E * ff * W)
        add("  like: gemm_dense", f"{E * W}x{ff} M={per}", T.us([lambda s, w=w: ck(lib.cmlb200_gemm_dense(w, fd.data_ptr(), ff, per, yw.data_ptr(), E * W, s)) for w in Dn], 4),
            2.0 * E * ff * W + per * (ff * 2.0 + E * W * 4), 2.0 * per * E * ff * W)


def run(pkg, synth, torch, peaks, sampler, kernels_only=False, models_only=False):
    out = {"latent": True, "data": "synthetic", "dtype": "bf16", "unit": "tok/s", "peaks": peaks,
           "config": {"prompts": PROMPTS, "new_tokens": NEW, "l2": "weights and caches of a step are larger than L2; decode kernels rotate over copies"}}
    sampler.start()
    if not models_only:
        out["kernels"] = kernel_table(pkg, synth, torch, peaks)
    if not kernels_only:
        out["4096_dense"] = {"sizes": {k: v for k, v in SIZES.items() if k != "batches"}, "latent_bf16": leg(pkg, synth, torch, dense_config(synth, SIZES), SIZES, peaks),
                             "grouped_bf16": layered_leg(pkg, synth, torch, GROUPED, peaks)}
        torch.cuda.empty_cache()
        out["2048_experts"] = {"sizes": {k: v for k, v in EXPERTS.items() if k != "batches"}, "latent_bf16": leg(pkg, synth, torch, mixed_config(synth, EXPERTS), EXPERTS, peaks)}
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
