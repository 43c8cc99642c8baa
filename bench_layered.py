"""Throughput of the layered models (`python bench.py --layered`) beside the framework's LLaMA at equal layer
sizes, and every kernel of both against its roofline. Random weights; all layers of a model file share one layer's
bytes on disk and are separate copies on the device. Not part of the default workload."""
import ctypes as C
import json
import tempfile
import time
from pathlib import Path

import numpy as np

# name -> layer sizes; "layers" keeps the files small, a step's weights are far larger than L2 all the same
MODELS = {
    "4096_mha": dict(vocab=32000, width=4096, heads=32, kv_heads=32, dim=128, ff=11008, layers=8, window=1024, batches=(1, 8, 32)),
    "8192_gqa": dict(vocab=32000, width=8192, heads=64, kv_heads=8, dim=128, ff=28672, layers=4, window=1024, batches=(1, 8, 32)),
}
PROMPTS, NEW = (512, 2048), 64


def model_sizes(c):
    per = c["width"] * c["dim"] * (2 * c["heads"] + 2 * c["kv_heads"]) + c["width"] * c["heads"] + 3 * c["width"] * c["ff"]
    return c["layers"] * per + c["vocab"] * c["width"], c["layers"] * per


def layered_leg(pkg, synth, torch, c, peaks):
    layer = lambda: synth.layered_layer(c["heads"], c["kv_heads"], c["dim"], c["dim"], c["window"], c["ff"], coef=0.1, every=512)
    cfg = synth.layered_config(c["vocab"], c["width"], [layer() for _ in range(c["layers"])])
    total, body = model_sizes(c)
    return model_leg(pkg, synth, torch, cfg, c, peaks, body, lambda B: total, lambda: 4 * c["layers"] * c["kv_heads"] * c["dim"])


def model_leg(pkg, synth, torch, cfg, c, peaks, body, weights, cache_bytes, row_bytes=0, weight=None):
    """Prefill and decode of a configuration with random weights. body: multiplications per token of a prompt. weights(B): those a
    decode step of B rows reads. cache_bytes(): read per row and cached token, all layers together (c["window"] of them).
    row_bytes: further bytes per row of a decode step (states). weight: (rng, name, shape) -> a tensor; the default suits designs
    whose norms are stored as they are."""
    rng = np.random.default_rng(5)
    out = {"weight_bytes": 2 * weights(max(c["batches"]))}
    with tempfile.TemporaryDirectory() as tmp:
        gen = lambda name, shape: (1 + 0.1 * rng.standard_normal(shape, dtype=np.float32)) if len(shape) == 1 else \
            rng.standard_normal(shape, dtype=np.float32) * np.float32(1.0 if name == "embed" else shape[1] ** -0.5)
        synth.write_layered(Path(tmp) / "m", cfg, (lambda name, shape: weight(rng, name, shape)) if weight else gen, alias_layers=True)
        nb = max(c["batches"])
        m = pkg.LanguageModel(Path(tmp) / "m", max_tokens=max(max(PROMPTS), nb * (c["window"] + NEW + 16)) + 64, max_sequences=nb, max_step_rows=4096)
    for n in PROMPTS:
        best = None
        for k in range(5):
            s = m.open()
            t = rng.integers(0, c["vocab"], n)
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            m.step([(s, t, [n - 1])], greedy=True)
            dt = time.perf_counter() - t0
            m.end(s)
            best = dt if k >= 2 and (best is None or dt < best) else best
        tf = 2.0 * body * n / best / 1e12
        out[f"prefill_{n}"] = {"tok_s": n / best, "ms": best * 1e3, "tflops_projections": tf, "frac_of_sustained": tf / peaks["bf16_tflops_sustained"]}
    for B in c["batches"]:
        seqs = [m.open() for _ in range(B)]
        ctx = c["window"]
        for s in seqs:
            m.step([(s, rng.integers(0, c["vocab"], ctx), [])])
        first = rng.integers(0, c["vocab"], B)
        m.decode_greedy(seqs, first, 8)
        _, ms = m.decode_greedy(seqs, first, NEW)
        for s in seqs:
            m.end(s)
        step = ms / NEW
        nbytes = 2 * weights(B) + B * (c["window"] * cache_bytes() + row_bytes)
        out[f"decode_b{B}"] = {"tok_s": B / (step * 1e-3), "ms_per_step": step, "gbs": nbytes / (step * 1e-3) / 1e9,
                               "frac_of_hbm": nbytes / (step * 1e-3) / 1e9 / peaks["hbm_gbs"]}
    m.close()
    return out


def llama_leg(pkg, synth, torch, c, peaks):
    """The same sizes as a Q4_0 LLaMA through cml_llama_*."""
    cfg = dict(vocab=c["vocab"], hidden=c["width"], inter=c["ff"], layers=c["layers"], heads=c["heads"], kv_heads=c["kv_heads"], max_seq=max(PROMPTS) + 64)
    total, body = model_sizes(c)
    out = {"weight_bytes": total * 18 // 32}
    path = Path(tempfile.gettempdir()) / "cmlb200_layered_bench.gguf"
    synth.write_random_llama_gguf(path, np.random.default_rng(99), cfg, alias_layers=True)
    nb = max(c["batches"])
    k = pkg.LlamaConfig(cfg["vocab"], cfg["hidden"], cfg["inter"], cfg["layers"], cfg["heads"], cfg["kv_heads"], cfg["max_seq"], 10000.0, 1e-5, 0, 0)
    m = pkg.lib.cml_llama_create(C.byref(k))
    assert m and pkg.lib.cml_llama_set_options(m, 0, nb) == 0 and pkg.lib.cml_llama_load_gguf(m, str(path).encode()) == 0
    path.unlink()
    rng = np.random.default_rng(7)
    for n in PROMPTS:
        best = None
        t = rng.integers(0, cfg["vocab"], n).astype(np.int32)
        for i in range(5):
            pkg.lib.cml_llama_reset(m)
            torch.cuda.synchronize()
            t0 = time.perf_counter()
            assert pkg.lib.cml_llama_prefill_sequence(m, 0, pkg.np_ptr(t), n) == 0
            dt = time.perf_counter() - t0
            best = dt if i >= 2 and (best is None or dt < best) else best
        tf = 2.0 * body * n / best / 1e12
        out[f"prefill_{n}"] = {"tok_s": n / best, "ms": best * 1e3, "tflops_projections": tf, "frac_of_sustained": tf / peaks["bf16_tflops_sustained"]}
    for B in c["batches"]:
        pkg.lib.cml_llama_reset(m)
        t = rng.integers(0, cfg["vocab"], (B, c["window"])).astype(np.int32)
        for b in range(B):
            assert pkg.lib.cml_llama_prefill_sequence(m, b, pkg.np_ptr(t[b]), c["window"]) == 0
        first, ids, ms = t[:, 0].copy(), np.zeros((NEW, B), np.int32), C.c_float(0)
        for _ in range(2):
            assert pkg.lib.cml_llama_decode_greedy(m, pkg.np_ptr(first), B, NEW, pkg.np_ptr(ids), C.byref(ms)) == 0
        step = ms.value / NEW
        nbytes = total * 18 / 32 + 2 * 2 * c["layers"] * B * (c["window"] + NEW) * c["kv_heads"] * c["dim"]
        out[f"decode_b{B}"] = {"tok_s": B / (step * 1e-3), "ms_per_step": step, "gbs": nbytes / (step * 1e-3) / 1e9,
                               "frac_of_hbm": nbytes / (step * 1e-3) / 1e9 / peaks["hbm_gbs"]}
    pkg.lib.cml_llama_free(m)
    return out


# ---- kernels -------------------------------------------------------------------------------------------------
class Timer:
    """us per launch of a list of closures (each with buffers of its own, together larger than L2), as one CUDA graph."""

    def __init__(self, torch):
        self.torch, self.stream = torch, torch.cuda.Stream()

    def us(self, calls, sweeps):
        torch = self.torch
        torch.cuda.synchronize()                       # the buffers were filled on another stream
        with torch.cuda.stream(self.stream):
            for f in calls:
                f(self.stream.cuda_stream)
            self.stream.synchronize()
            g = torch.cuda.CUDAGraph()
            with torch.cuda.graph(g, stream=self.stream, capture_error_mode="thread_local"):
                for _ in range(sweeps):
                    for f in calls:
                        f(self.stream.cuda_stream)
            for _ in range(3):
                g.replay()
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record(self.stream)
            for _ in range(5):
                g.replay()
            e1.record(self.stream)
            e1.synchronize()
        return e0.elapsed_time(e1) * 1e3 / (5 * sweeps * len(calls))


def copies_for(nbytes):
    return max(2, int(300e6 // max(nbytes, 1)) + 1) if nbytes < 300e6 else 2


def kernel_table(pkg, synth, torch, peaks):
    """One line per kernel of the layered path with the like kernel of the LLaMA path under it."""
    dev, lib, T, out = torch.device("cuda:0"), pkg.lib, Timer(torch), []
    ck = pkg.check
    rng = np.random.default_rng(3)

    def add(kernel, shape, us, nbytes=None, flops=None):
        if flops:
            a, p, u = flops / us / 1e6, peaks["bf16_tflops"], "TFLOP/s"
        else:
            a, p, u = nbytes / us / 1e3, peaks["hbm_gbs"], "GB/s"
        out.append({"kernel": kernel, "shape": shape, "us": round(us, 2), "achieved": round(a, 1), "unit": u, "frac": round(a / p, 3)})

    def q4(N, K, n):
        ws = []
        for _ in range(n):
            qs = torch.randint(0, 256, (N * K // 2,), device=dev, dtype=torch.uint8)
            sc = (torch.rand(N * K // 32, device=dev) * 1e-2 + 1e-3).half()
            ws.append((pkg.QMat(pkg.Q4_0, N, K, 32, qs.data_ptr(), sc.data_ptr(), 0, None), qs, sc))
        return ws

    for N, K in ((4096, 4096), (22016, 4096), (4096, 11008), (8192, 28672), (32000, 4096)):
        glu = N == 22016
        n = copies_for(2 * N * K)
        w = [torch.randn(N, K, device=dev).mul_(K ** -0.5).bfloat16() for _ in range(n)]
        W = [pkg.Dense(pkg.DT_BF16, N, K, K, t.data_ptr()) for t in w]
        for M in (1, 8, 32):
            x = torch.randn(M, K, device=dev).bfloat16()
            y = torch.empty(M, N, device=dev)
            if glu:
                calls = [lambda s, d=d: ck(lib.cmlb200_gemv_dense_glu(d, x.data_ptr(), K, M, N // 2, pkg.ACT_GELU_TANH, y.data_ptr(), N // 2, s)) for d in W]
            else:
                calls = [lambda s, d=d: ck(lib.cmlb200_gemv_dense(d, x.data_ptr(), K, M, y.data_ptr(), N, s)) for d in W]
            add("gemv_dense" + ("_glu" if glu else ""), f"{N}x{K} M={M}", T.us(calls, 4), nbytes=2 * N * K + M * K * 2 + M * N * (1 if glu else 4))
        for M in (64, 512, 2048):
            x = torch.randn(M, K, device=dev).bfloat16()
            y = torch.empty(M, N, device=dev)
            if glu:
                calls = [lambda s, d=d: ck(lib.cmlb200_gemm_dense_glu(d, x.data_ptr(), K, M, N // 2, pkg.ACT_GELU_TANH, y.data_ptr(), N // 2, s)) for d in W]
            else:
                calls = [lambda s, d=d: ck(lib.cmlb200_gemm_dense(d, x.data_ptr(), K, M, y.data_ptr(), N, s)) for d in W]
            us = T.us(calls, 2)
            small = M == 64
            add("gemm_dense" + ("_glu" if glu else ""), f"{N}x{K} M={M}", us, nbytes=2 * N * K + 2 * M * K + M * N * (1 if glu else 4) if small else None,
                flops=None if small else 2.0 * M * N * K)
        del w, W
        torch.cuda.empty_cache()
        if glu:
            continue
        ws = q4(N, K, copies_for(N * K * 18 // 32))
        for M in (1, 8, 32):
            x, y = torch.randn(M, K, device=dev), torch.empty(M, N, device=dev)
            calls = [lambda s, q=q: ck(lib.cmlb200_gemv(C.byref(q[0]), x.data_ptr(), y.data_ptr(), M, s)) for q in ws]
            add("  llama gemv q4_0", f"{N}x{K} M={M}", T.us(calls, 4), nbytes=N * K * 18 / 32 + M * K * 4 + M * N * 4)
        for M in (64, 512, 2048):
            x, y = torch.randn(M, K, device=dev).bfloat16(), torch.empty(M, N, device=dev, dtype=torch.bfloat16)
            calls = [lambda s, q=q: ck(lib.cmlb200_gemm_bf16(C.byref(q[0]), x.data_ptr(), y.data_ptr(), M, s)) for q in ws]
            us = T.us(calls, 2)
            add("  llama gemm q4_0", f"{N}x{K} M={M}", us, nbytes=N * K * 18 / 32 + 2 * M * K + 2 * M * N if M == 64 else None,
                flops=None if M == 64 else 2.0 * M * N * K)
        del ws
        torch.cuda.empty_cache()
    attention_rows(pkg, torch, T, add, rng)
    for rows, dim in ((1, 4096), (8, 4096), (512, 4096), (2048, 8192)):
        n = copies_for(rows * dim * 14)
        xs = [torch.randn(rows, dim, device=dev) for _ in range(min(n, 64))]
        y, h = torch.randn(rows, dim, device=dev), torch.empty(rows, dim, device=dev, dtype=torch.bfloat16)
        w1, w2, w16 = torch.ones(dim, device=dev), torch.ones(dim, device=dev), torch.ones(dim, device=dev).half()
        calls = [lambda s, x=x: ck(lib.cmlb200_residual_norm(x.data_ptr(), y.data_ptr(), dim, w1.data_ptr(), w2.data_ptr(), 1e-5, rows, dim, None, h.data_ptr(),
                                                             pkg.DT_BF16, dim, s)) for x in xs]
        add("residual_norm", f"{rows}x{dim}", T.us(calls, 4), nbytes=rows * dim * 14)
        calls = [lambda s, x=x: ck(lib.cmlb200_rmsnorm(x.data_ptr(), w16.data_ptr(), rows, dim, 1e-5, None, h.data_ptr(), s)) for x in xs]
        add("  llama rmsnorm", f"{rows}x{dim}", T.us(calls, 4), nbytes=rows * dim * 6)
    tab, x = torch.randn(32000, 4096, device=dev), None
    fr = torch.rand(2049, device=dev)
    tb, th = tab.bfloat16(), tab.half()
    for rows in (1, 2048):
        tok, pos, x = torch.randint(0, 32000, (rows,), device=dev, dtype=torch.int32), torch.arange(rows, device=dev, dtype=torch.int32), torch.empty(rows, 4096, device=dev)
        add("embed_rows", f"{rows}x4096", T.us([lambda s: ck(lib.cmlb200_embed_rows(tb.data_ptr(), pkg.DT_BF16, tok.data_ptr(), pos.data_ptr(), fr.data_ptr(), rows, 4096,
                                                                                 32000, x.data_ptr(), s))], 32), nbytes=rows * 4096 * 6)
        add("  llama embed_f16", f"{rows}x4096", T.us([lambda s: ck(lib.cmlb200_embed_f16(th.data_ptr(), tok.data_ptr(), rows, 4096, 32000, x.data_ptr(), s))], 32),
            nbytes=rows * 4096 * 6)
    return out


def attention_rows(pkg, torch, T, add, rng):
    dev, lib, ck = torch.device("cuda:0"), pkg.lib, pkg.check
    for H, G, D in ((32, 32, 128), (64, 8, 128)):
        slopes = torch.tensor([2.0 ** (-8 * (h + 1) / H) for h in range(H)], device=dev)
        qn, kn = torch.ones(H * D, device=dev), torch.ones(G * D, device=dev)
        ld = H * D + 2 * G * D + H
        # decode: B rows of `ctx` cached keys
        for B, ctx in ((1, 1024), (8, 1024), (32, 1024)):
            per = ctx // 16 + 1
            n = copies_for(4 * B * ctx * G * D)
            n = min(n, 24)
            table = torch.arange(B * per, device=dev, dtype=torch.int32).view(B, per).contiguous()
            qkv = torch.randn(B, ld, device=dev)
            pos, slot = torch.full((B,), ctx, device=dev, dtype=torch.int32), torch.arange(B, device=dev, dtype=torch.int32)
            pools = [(torch.randn(B * per * 16, G, D, device=dev).half(), torch.randn(B * per * 16, G, D, device=dev).half()) for _ in range(n)]
            att = [pkg.Attn(H, G, D, D, D, D, D ** -0.5, 0, slopes.data_ptr(), 1, qn.data_ptr(), kn.data_ptr(), 1e-5, 0.1, 512.0, ld - H, pkg.DT_F16, k.data_ptr(),
                            v.data_ptr(), 16, table.data_ptr(), per) for k, v in pools]
            o = torch.empty(B, H * D, device=dev, dtype=torch.bfloat16)
            calls = [lambda s, a=a: ck(lib.cmlb200_attention_one(a, qkv.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), B, ctx, o.data_ptr(), H * D, s)) for a in att]
            add("attention_one", f"H={H} G={G} B={B} ctx={ctx}", T.us(calls, 8), nbytes=4 * B * ctx * G * D)
            del pools
            pools = [(torch.randn(B, ctx + 32, G * D, device=dev).half(), torch.randn(B, ctx + 32, G * D, device=dev).half()) for _ in range(n)]
            splits = (ctx + 32) // 32
            scr = torch.zeros(lib.cmlb200_attention_decode_scratch_bytes(B, H, D, splits) // 4 + 16, device=dev)
            cs, of = torch.zeros(B, D, device=dev), torch.empty(B, H * D, device=dev)
            calls = [lambda s, k=k, v=v: ck(lib.cmlb200_attention_decode(qkv.data_ptr(), ld, k.data_ptr(), v.data_ptr(), slot.data_ptr(), pos.data_ptr(), pos.data_ptr(), B,
                                                                         H, G, D, ctx + 32, ctx, 0, cs.data_ptr(), of.data_ptr(), scr.data_ptr(), splits, s)) for k, v in pools]
            add("  llama attention_decode", f"H={H} G={G} B={B} ctx={ctx}", T.us(calls, 8), nbytes=4 * B * ctx * G * D)
            del pools
            torch.cuda.empty_cache()
        for n in (512, 2048):
            for window in (0, 256):
                per = n // 16
                k, v = (torch.randn(n, G, D, device=dev).half() for _ in range(2))
                table = torch.arange(per, device=dev, dtype=torch.int32).view(1, per)
                qkv, o = torch.randn(n, ld, device=dev), torch.empty(n, H * D, device=dev, dtype=torch.bfloat16)
                tiles = torch.tensor([[i, 64, 0, i] for i in range(0, n, 64)], device=dev, dtype=torch.int32)
                pos, slot = torch.arange(n, device=dev, dtype=torch.int32), torch.zeros(n, device=dev, dtype=torch.int32)
                a = pkg.Attn(H, G, D, D, D, D, D ** -0.5, window, slopes.data_ptr(), 1, qn.data_ptr(), kn.data_ptr(), 1e-5, 0.1, 512.0, ld - H, pkg.DT_F16, k.data_ptr(),
                             v.data_ptr(), 16, table.data_ptr(), per)
                pairs = n * (n + 1) / 2 if not window else n * window - window * (window - 1) / 2
                add("attention_tiles", f"H={H} G={G} rows={n} window={window}",
                    T.us([lambda s: ck(lib.cmlb200_attention_tiles(a, qkv.data_ptr(), ld, tiles.data_ptr(), len(tiles), o.data_ptr(), H * D, s))], 10), flops=4.0 * pairs * H * D)
                if not window:
                    add("qk_norm_append", f"H={H} G={G} rows={n}",
                        T.us([lambda s: ck(lib.cmlb200_qk_norm_append(a, qkv.data_ptr(), ld, pos.data_ptr(), slot.data_ptr(), n, s))], 10),
                        nbytes=n * (H * D * 8 + G * D * 8 + 4 * G * D))
                    k2, v2 = k.view(n, G * D), v.view(n, G * D)
                    add("  llama attention_prefill", f"H={H} G={G} rows={n}",
                        T.us([lambda s: ck(lib.cmlb200_attention_prefill(qkv.data_ptr(), ld, k2.data_ptr(), v2.data_ptr(), 0, pos.data_ptr(), n, H, G, D, n, None, o.data_ptr(),
                                                                         s))], 10), flops=4.0 * pairs * H * D)
                    q2 = torch.randn(n, ld, device=dev)
                    add("  llama qkv_rope_append", f"H={H} G={G} rows={n}",
                        T.us([lambda s: ck(lib.cmlb200_qkv_rope_append(q2.data_ptr(), ld, slot.data_ptr(), pos.data_ptr(), n, H, G, D, 10000.0, H, k2.data_ptr(), v2.data_ptr(), n,
                                                                      0, s))], 10), nbytes=n * (H * D * 8 + G * D * 8 + 4 * G * D))


def run(pkg, synth, torch, peaks, sampler, kernels_only=False, models_only=False):
    out = {"layered": True, "data": "synthetic", "dtype": "bf16", "unit": "tok/s", "peaks": peaks,
           "config": {"prompts": PROMPTS, "new_tokens": NEW, "l2": "weights and caches of a step are larger than L2; kernels rotate over copies"}}
    sampler.start()
    if not models_only:
        out["kernels"] = kernel_table(pkg, synth, torch, peaks)
    if not kernels_only:
        for name, c in MODELS.items():
            out[name] = {"sizes": {k: v for k, v in c.items() if k != "batches"}, "layered_bf16": layered_leg(pkg, synth, torch, c, peaks),
                         "llama_q4_0": llama_leg(pkg, synth, torch, c, peaks)}
            torch.cuda.empty_cache()
    out["clocks"] = sampler.stop()
    print(json.dumps(out))
