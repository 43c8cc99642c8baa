"""Seeded synthetic inputs with the shapes and value distributions of the benchmark configs
(numpy only; shared by tests/ and bench.py). Nothing here computes results."""
import numpy as np


def q8_0_blocks(rng, rows, cols, d_lo=1e-3, d_hi=1e-2):
    """GGUF Q8_0 blocks, file order: int8 uniform in [-127,127], fp16 d uniform in [d_lo,d_hi]."""
    nb = rows * cols // 32
    blk = np.empty((nb, 34), np.uint8)
    blk[:, :2] = rng.uniform(d_lo, d_hi, nb).astype(np.float16).view(np.uint8).reshape(nb, 2)
    blk[:, 2:] = rng.integers(-127, 128, (nb, 32), dtype=np.int8).view(np.uint8)
    return blk.reshape(-1)


def q4_0_blocks(rng, rows, cols, d_lo=1e-3, d_hi=2e-2):
    """GGUF Q4_0 blocks: nibbles uniform 0..15, fp16 d uniform in [d_lo,d_hi]."""
    nb = rows * cols // 32
    blk = np.empty((nb, 18), np.uint8)
    blk[:, :2] = rng.uniform(d_lo, d_hi, nb).astype(np.float16).view(np.uint8).reshape(nb, 2)
    blk[:, 2:] = rng.integers(0, 256, (nb, 16), dtype=np.uint8)
    return blk.reshape(-1)


GGUF_BLOCK = {2: (32, 18), 3: (32, 20), 7: (32, 34), 12: (256, 144), 13: (256, 176), 14: (256, 210)}   # type -> (elements, bytes)


def gguf_blocks(rng, gtype, rows, cols, std=0.02):
    """Random GGUF blocks of type Q4_1 (3), Q4_K (12), Q5_K (13) or Q6_K (14) in C-ML's layouts
    (src/core/gguf_quant.c:90-311) whose dequantised weights have mean about 0 and roughly `std`:
    uniform quants, small integer sub-block scales, fp16 d / dmin / m chosen to centre the values."""
    if gtype == 2: return q4_0_blocks(rng, rows, cols, std / 6, std / 3)
    if gtype == 7: return q8_0_blocks(rng, rows, cols, std / 100, std / 50)
    be, bb = GGUF_BLOCK[gtype]
    nb = rows * cols // be
    blk = rng.integers(0, 256, (nb, bb), dtype=np.uint8)
    f16 = lambda a: np.asarray(a, np.float16).view(np.uint8).reshape(nb, 2)
    if gtype == 3:                                   # w = q * d + m, q uniform 0..15
        d = rng.uniform(0.5, 1.0, nb) * std / 4.6
        blk[:, 0:2] = f16(d)
        blk[:, 2:4] = f16(-7.5 * d * rng.uniform(0.9, 1.1, nb))
    elif gtype in (12, 13):                          # w = q * (d * sc) - dmin * mn, q uniform 0..15 (0..31)
        qmax = 15 if gtype == 12 else 31
        sc = rng.integers(2, 8 if gtype == 12 else 4, (nb, 8))
        mn = np.clip(np.rint(qmax / 2 * sc + rng.integers(-2, 3, (nb, 8))), 0, 63).astype(np.int64)
        s = np.zeros((nb, 12), np.int64)             # get_scale_min_k4's packing
        s[:, 0:4] = sc[:, 0:4] | ((sc[:, 4:8] >> 4) << 6)
        s[:, 4:8] = mn[:, 0:4] | ((mn[:, 4:8] >> 4) << 6)
        s[:, 8:12] = (sc[:, 4:8] & 15) | ((mn[:, 4:8] & 15) << 4)
        d = rng.uniform(0.5, 1.0, nb) * std / (5.0 * (qmax + 1) / 3.46)
        blk[:, 0:2] = f16(d)
        blk[:, 2:4] = f16(d)
        blk[:, 4:16] = s.astype(np.uint8)
    else:                                            # w = d * scale8 * (q - 32), q uniform 0..63
        blk[:, 192:208] = rng.integers(-24, 25, (nb, 16)).astype(np.int8).view(np.uint8)
        blk[:, 208:210] = f16(rng.uniform(0.5, 1.0, nb) * std / (14.0 * 18.5))
    return blk.reshape(-1)


def nf4_weight(rng, rows, cols, block=64, s_lo=0.01, s_hi=0.1):
    """NF4 packed bytes (indices uniform 0..15) and fp32 absmax per block of the flat index."""
    packed = rng.integers(0, 256, rows * cols // 2, dtype=np.uint8)
    scales = rng.uniform(s_lo, s_hi, rows * cols // block).astype(np.float32)
    return packed, scales


def bf16_round(a):
    """fp32 -> nearest-even bf16, returned both as uint16 bit patterns and as fp32 values."""
    u = np.ascontiguousarray(a, np.float32).view(np.uint32).astype(np.uint64)
    r = ((u + 0x7FFF + ((u >> 16) & 1)) >> 16).astype(np.uint16)
    return r, (r.astype(np.uint32) << 16).view(np.float32)


def bf16_to_f32(u16):
    return (np.ascontiguousarray(u16, np.uint16).astype(np.uint32) << 16).view(np.float32)


# ---- GGUF v3 writer for synthetic models (little-endian; tensor data 32-byte aligned) ------------
_GGUF_SCALAR = {0: "<B", 1: "<b", 2: "<H", 3: "<h", 4: "<I", 5: "<i", 6: "<f", 7: "<B", 10: "<Q", 11: "<q", 12: "<d"}


def _gguf_value(vtype, value):
    """One GGUF metadata value: scalars by type id, 8 = string (bytes or str), 9 = (elem_type, items)."""
    import struct
    if vtype == 8:
        raw = value.encode() if isinstance(value, str) else bytes(value)
        return struct.pack("<Q", len(raw)) + raw
    if vtype == 9:
        et, items = value
        return struct.pack("<IQ", et, len(items)) + b"".join(_gguf_value(et, v) for v in items)
    return struct.pack(_GGUF_SCALAR[vtype], value)


def write_gguf(path, tensors, metadata=None):
    """tensors: list of (name, dims, gguf_type, raw_bytes). dims are written in the given order
    (for weights: (in_features, out_features), the GGUF convention). metadata: list of
    (key, value_type, value) written after general.architecture = "llama"."""
    import struct
    infos, blobs, off = [], [], 0
    for name, dims, gtype, raw in tensors:
        raw = bytes(raw)
        infos.append((name.encode(), dims, gtype, off))
        pad = (-len(raw)) % 32
        blobs.append(raw + b"\0" * pad)
        off += len(raw) + pad
    out = bytearray()
    metadata = list(metadata or [])
    out += struct.pack("<IIQQ", 0x46475547, 3, len(tensors), 1 + len(metadata))
    key = b"general.architecture"
    out += struct.pack("<Q", len(key)) + key + struct.pack("<I", 8) + struct.pack("<Q", 5) + b"llama"
    for k, vtype, value in metadata:
        k = k.encode() if isinstance(k, str) else bytes(k)
        out += struct.pack("<Q", len(k)) + k + struct.pack("<I", vtype) + _gguf_value(vtype, value)
    for name, dims, gtype, o in infos:
        out += struct.pack("<Q", len(name)) + name + struct.pack("<I", len(dims))
        for d in dims:
            out += struct.pack("<Q", d)
        out += struct.pack("<IQ", gtype, o)
    out += b"\0" * ((-len(out)) % 32)
    with open(path, "wb") as f:
        f.write(out)
        for b in blobs:
            f.write(b)


def make_llama(rng, cfg, quantize, qtype=2, wscale=0.05):
    """Random LLaMA weights quantized with `quantize(fp32 [out,in]) -> GGUF block bytes`.
    Returns (gguf tensor list, dict of quantized block arrays + fp16 vectors)."""
    V, H, I, L = cfg["vocab"], cfg["hidden"], cfg["inter"], cfg["layers"]
    hd = H // cfg["heads"]
    QW, KVW = cfg["heads"] * hd, cfg["kv_heads"] * hd
    tensors, store = [], {}

    def proj(name, out_f, in_f):
        w = (rng.standard_normal((out_f, in_f)) * wscale).astype(np.float32)
        blocks = quantize(w)
        store[name] = (blocks, out_f, in_f)
        tensors.append((name, (in_f, out_f), qtype, blocks.tobytes()))

    def vec(name, n, base=1.0, rows=None):
        shape = (rows, n) if rows else (n,)
        v = (base + 0.1 * rng.standard_normal(shape)).astype(np.float16) if base else (rng.standard_normal(shape) * 0.5).astype(np.float16)
        store[name] = v
        tensors.append((name, tuple(reversed(shape)), 1, v.tobytes()))

    vec("token_embd.weight", H, base=0.0, rows=V)
    for l in range(L):
        vec(f"blk.{l}.attn_norm.weight", H)
        proj(f"blk.{l}.attn_q.weight", QW, H)
        proj(f"blk.{l}.attn_k.weight", KVW, H)
        proj(f"blk.{l}.attn_v.weight", KVW, H)
        proj(f"blk.{l}.attn_output.weight", H, QW)
        vec(f"blk.{l}.ffn_norm.weight", H)
        proj(f"blk.{l}.ffn_gate.weight", I, H)
        proj(f"blk.{l}.ffn_up.weight", I, H)
        proj(f"blk.{l}.ffn_down.weight", H, I)
    vec("output_norm.weight", H)
    proj("output.weight", V, H)
    return tensors, store


def write_random_llama_gguf(path, rng, cfg, qtype=2, weight_std=0.02, alias_layers=False):
    """A LLaMA-shaped GGUF with random Q4_0/Q8_0 blocks (uniform quants, fp16 scales chosen so
    that the dequantised weights have roughly `weight_std`), fp16 norms near 1 and fp16
    embeddings. Generated tensor by tensor straight into the file, so 7B-sized models need no
    fp32 staging; every layer reuses the random bytes drawn for layer 0. By default the file
    still holds each layer separately; with alias_layers the tensor infos of layers 1.. point at
    layer 0's data (GGUF addresses tensors by offset, so this is a valid file of a fraction of
    the size; the loader still uploads every layer as its own device copy). Returns the number
    of bytes written."""
    import struct
    V, H, I, L = cfg["vocab"], cfg["hidden"], cfg["inter"], cfg["layers"]
    hd = H // cfg["heads"]
    QW, KVW = cfg["heads"] * hd, cfg["kv_heads"] * hd
    bb, qstd = (18, 4.6) if qtype == 2 else (34, 73.0)
    d0 = weight_std / qstd
    spec = [("token_embd.weight", (H, V), 1)]
    for l in range(L):
        spec += [(f"blk.{l}.attn_norm.weight", (H,), 1), (f"blk.{l}.attn_q.weight", (H, QW), qtype),
                 (f"blk.{l}.attn_k.weight", (H, KVW), qtype), (f"blk.{l}.attn_v.weight", (H, KVW), qtype),
                 (f"blk.{l}.attn_output.weight", (QW, H), qtype), (f"blk.{l}.ffn_norm.weight", (H,), 1),
                 (f"blk.{l}.ffn_gate.weight", (H, I), qtype), (f"blk.{l}.ffn_up.weight", (H, I), qtype),
                 (f"blk.{l}.ffn_down.weight", (I, H), qtype)]
    spec += [("output_norm.weight", (H,), 1), ("output.weight", (H, V), qtype)]

    def nbytes(dims, t):
        n = int(np.prod(dims))
        return n * 2 if t == 1 else n // 32 * bb

    def kind_of(name, dims, t):
        return (name.split(".", 2)[2] if name.startswith("blk.") else name, dims, t)

    head = bytearray(struct.pack("<IIQQ", 0x46475547, 3, len(spec), 0))
    off = 0
    placed = {}         # alias_layers: data offset of the first tensor of each kind
    stored = []         # the tensors whose bytes go into the file, in order
    for name, dims, t in spec:
        nb = name.encode()
        head += struct.pack("<Q", len(nb)) + nb + struct.pack("<I", len(dims))
        for d in dims:
            head += struct.pack("<Q", d)
        kind = kind_of(name, dims, t)
        if alias_layers and kind in placed:
            head += struct.pack("<IQ", t, placed[kind])
            continue
        placed[kind] = off
        stored.append((name, dims, t))
        head += struct.pack("<IQ", t, off)
        off += (nbytes(dims, t) + 31) // 32 * 32
    head += b"\0" * ((-len(head)) % 32)
    cache = {}          # layers share their random bytes: one draw per (tensor kind, shape)
    with open(path, "wb") as f:
        f.write(head)
        for name, dims, t in stored:
            n = int(np.prod(dims))
            kind = kind_of(name, dims, t)
            if kind in cache:
                raw = cache[kind]
            elif t == 1:
                if len(dims) == 1:
                    raw = (1.0 + 0.05 * rng.standard_normal(n)).astype(np.float16).tobytes()
                else:
                    raw = (0.5 * rng.standard_normal(n, dtype=np.float32)).astype(np.float16).tobytes()
            else:
                nblk = n // 32
                blk = np.empty((nblk, bb), np.uint8)
                blk[:, :2] = rng.uniform(0.5 * d0, 1.5 * d0, nblk).astype(np.float16).view(np.uint8).reshape(nblk, 2)
                blk[:, 2:] = rng.integers(0, 256, (nblk, bb - 2), dtype=np.uint8)
                raw = blk.tobytes()
            cache[kind] = raw
            f.write(raw)
            f.write(b"\0" * ((-len(raw)) % 32))
    return len(head) + off


# ---- layered models: a folder with config.json and model.safetensors --------------------------------
def layered_layer(heads, kv_heads, dim, vdim, window, ff, scale=None, coef=0.2, every=50, weights_of=None):
    layer = {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5,
                                            "mask": {"size": window}, "q_temp": {"coef": coef, "every": every}},
             "mlp": {"kind": "dense", "ff": ff} if ff else None}
    if weights_of is not None:
        layer["weights_of"] = weights_of
    return layer


def layered_config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Rarolorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def latent_layer(heads, dim, rot_dim, vdim, rank, mlp, window=None, gated=False, base=10000.0, scaling=None, scale=None, kv_from=None):
    """mlp: a dense layer's size, (experts, top, size, limit), or None. scaling: (factor, original, fast, slow)."""
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "original", "fast", "slow"), scaling))
    mixer = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "rot": rot, "scale": scale or (dim + rot_dim) ** -0.5}
    if window:
        mixer["mask"] = {"size": window}
    if kv_from is not None:
        mixer["kv_from"] = kv_from
    if isinstance(mlp, tuple):
        mlp = {"kind": "moe", "router": {"experts": mlp[0], "top": mlp[1]}, "expert": {"ff": mlp[2], "limit": mlp[3]}}
    elif mlp:
        mlp = {"kind": "dense", "ff": mlp}
    return {"type": "latent_attention_2" if gated else "latent_attention", "mixer": mixer, "mlp": mlp or None}


def latent_config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Situlorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


def latent_layer_shapes(layer, W, p):
    m, f = layer["mixer"], layer["mlp"]
    H, R = m["heads"], m["kv_rank"]
    out = {p + "norm1": (W,), p + "mix.q": (H * (m["dim"] + m["rot_dim"]), W), p + "mix.uk": (H * m["dim"], R), p + "mix.uv": (H * m["vdim"], R),
           p + "mix.o": (W, H * m["vdim"])}
    if m.get("kv_from") is None:
        out.update({p + "mix.dkv": (R + m["rot_dim"], W), p + "mix.dkv.norm": (R,)})
    if layer["type"] == "latent_attention_2":
        out[p + "mix.g"] = (H * m["vdim"], W)
    if f:
        out[p + "norm2"] = (W,)
        if f["kind"] == "dense":
            out.update({p + "mlp.up": (f["ff"], W), p + "mlp.down": (W, f["ff"]), p + "mlp.act": (4,)})
        else:
            n = f["expert"]["ff"]
            out[p + "mlp.router"] = (f["router"]["experts"], W)
            for e in range(f["router"]["experts"]):
                out.update({p + f"mlp.e{e}.gate": (n, W), p + f"mlp.e{e}.up": (n, W), p + f"mlp.e{e}.down": (W, n)})
    return out


def routed_mlp(experts, identity, top, groups, keep, ff, shared, scale=1.5):
    return {"kind": "moe", "expert": {"ff": ff}, "shared": {"ff": shared},
            "router": {"experts": experts, "identity": identity, "top": top, "groups": {"count": groups, "keep": keep}, "scale": scale}}


def kept_layer(heads, kv_heads, dim, window, keep, mlp, scale=None):
    """mlp: a dense layer's size, routed_mlp(..), or None."""
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale or dim ** -0.5,
                                           "mask": {"size": window, "keep_first": keep}},
            "mlp": {"kind": "dense", "ff": mlp} if isinstance(mlp, int) else mlp}


def parallel_layer(left, right, ranks, mlp, scales=(0.8, 1.3)):
    """left: (heads, kv_heads, dim, vdim, chunk), right: (heads, kv_heads, dim, vdim, taps), ranks: of the decay's and the gate's projections
    (these only shape tensors)."""
    lm = dict(zip(("heads", "kv_heads", "dim", "vdim"), left), scale=left[2] ** -0.5, mask={"size": left[4]})
    return {"type": "parallel", "mixer": {"left": lm, "left_scale": scales[0], "right": dict(zip(("heads", "kv_heads", "dim", "vdim", "conv"), right)), "right_scale": scales[1]},
            "mlp": {"kind": "dense", "ff": mlp} if isinstance(mlp, int) else mlp, "ranks": list(ranks)}


def streams_config(vocab, width, streams, layers, eps=1e-5, scale=2.0, cap=6.0):
    return {"architecture": "Lenedra", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps}, "embedding": {"scale": scale},
            "logit_softcap": cap, "layers": layers}


def streams_layer_shapes(layer, W, streams, p):
    m, f, out = layer["mixer"], layer["mlp"], {}

    def sublayer(n):
        out.update({p + f"norm{n}": (W,), p + f"hc{n}.in": (streams,), p + f"hc{n}.out": (streams,), p + f"hc{n}.mix": (streams, streams)})

    def projections(q, pairs):
        for name, rows in pairs:
            out.update({q + name: (rows, W), q + name + ".b": (rows,)})
    sublayer(1)
    if layer["type"] == "attention":
        H, G, D, q = m["heads"], m["kv_heads"], m["dim"], p + "mix."
        projections(q, (("q", H * D), ("k", G * D)))
        out.update({q + "q.norm": (D,), q + "k.norm": (D,), q + "o": (W, H * D), q + "o.b": (W,)})
    else:
        a, r, q = m["left"], m["right"], p + "mix.left."
        projections(q, (("q", a["heads"] * a["dim"]), ("k", a["kv_heads"] * a["dim"]), ("v", a["kv_heads"] * a["vdim"])))
        out.update({q + "sink": (a["heads"],), q + "o": (W, a["heads"] * a["vdim"])})
        H, qk, v, q = r["heads"], r["kv_heads"] * r["dim"], r["heads"] * r["vdim"], p + "mix.right."
        for name, rows in (("q", qk), ("k", qk), ("v", v)):
            out.update({q + name: (rows, W), q + name + ".conv": (rows, r["conv"])})
        ra, rg = layer["ranks"]
        out.update({q + "b": (H, W), q + "A_log": (H,), q + "dt_bias": (H * r["dim"],), q + "norm": (r["vdim"],), q + "a1": (ra, W), q + "a2": (H * r["dim"], ra),
                    q + "g1": (rg, W), q + "g2": (v, rg), q + "o": (W, v)})
    if not f:
        return out
    sublayer(2)

    def gated(q, n):
        out.update({q + "gate": (n, W), q + "up": (n, W), q + "down": (W, n)})
    if f["kind"] == "dense":
        gated(p + "mlp.", f["ff"])
        return out
    n = f["router"]["experts"] + f["router"]["identity"]
    out.update({p + "mlp.router": (n, W), p + "mlp.correction": (n,)})
    for e in range(f["router"]["experts"]):
        gated(p + f"mlp.e{e}.", f["expert"]["ff"])
    gated(p + "mlp.shared.", f["shared"]["ff"])
    return out


def streams_weight(rng, name, shape):
    """A random tensor of a design with streams: decays between nearly none and nearly all, sinks that take a visible share,
    streams that mix, corrections in widely separated steps."""
    a = rng.standard_normal(shape).astype(np.float32)
    leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
    if leaf.startswith("norm") or leaf == "final.norm":
        a *= 0.2
    elif leaf.endswith(".norm"):
        a = 1 + 0.2 * a
    elif leaf.endswith((".q.b", ".k.b", ".v.b", ".o.b")):
        a *= 0.3
    elif leaf.endswith(".sink"):
        a += 1
    elif leaf.endswith(".A_log"):
        a = rng.uniform(-4, 1, shape)
    elif leaf.endswith(".dt_bias"):
        a -= 1
    elif leaf.endswith(".correction"):
        a = rng.choice([0.75, -1.5, -3.75], shape)
    elif leaf.startswith("hc"):
        a = 0.15 * a + (np.eye(shape[0]) if len(shape) == 2 else 0.7)
    elif leaf != "embed":
        a /= np.sqrt(shape[-1])
    return bf16_round(np.asarray(a, np.float32))[1]


def sigmoid_mlp(experts, top, ff, groups=None):
    """Experts without a gate; groups: (count, keep)."""
    router = {"experts": experts, "top": top}
    if groups:
        router["groups"] = dict(zip(("count", "keep"), groups))
    return {"kind": "moe", "expert": {"ff": ff}, "router": router}


def _rotation(dims, base, keys, scaling):
    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(keys, scaling))
    return rot


def talking_layer(heads, kv_heads, dim, vdim, window, taps, cap, mlp, rot, scaling=None, scale=None):
    """rot: (dims, base), scaling: (factor, low, high, original)."""
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": window}, "conv": taps, "softcap": cap,
                                                       "scale": scale or dim ** -0.5, "rot": _rotation(*rot, ("factor", "low", "high", "original"), scaling)}}


def queried_layer(heads, dim, rot_dim, vdim, q_rank, kv_rank, mlp, base=10000.0, scale=None):
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                                                              "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": base}}}


def recurrent_layer(left, rot, width, mlp, factor=None, scale=None):
    """left: (heads, kv_heads, dim, vdim, window), rot: (dims, base)."""
    m = dict(zip(("heads", "kv_heads", "dim", "vdim"), left), mask={"size": left[4]}, scale=scale or left[2] ** -0.5, rot=_rotation(*rot, ("factor",), factor and (factor,)))
    return {"type": "parallel", "mlp": mlp, "mixer": {"left": m, "right": {"width": width}}}


def looped_config(vocab, width, layers, loop=None, eps=1e-5):
    """loop: (start, stop, times)."""
    cfg = {"architecture": "Zevilorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    return cfg


def gated_layer_shapes(layer, W, p):
    m, f, q = layer["mixer"], layer["mlp"], p + "mix."
    out = {p + "norm1": (W,), p + "rg1": (W, W), p + "rg1.b": (W,)}
    if layer["type"] == "attention":
        H, G, D, V, n = m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["conv"]
        for name, rows in (("q", H * D), ("k", G * D), ("v", G * V)):
            out.update({q + name: (rows, W), q + name + ".b": (rows,), q + name + ".conv": (rows, n)})
        out.update({q + "talk": (H, H), q + "o": (W, H * V), q + "o.b": (W,)})
    elif layer["type"] == "latent_attention":
        H, R = m["heads"], m["kv_rank"]
        out.update({q + "dq": (m["q_rank"], W), q + "dq.norm": (m["q_rank"],), q + "uq": (H * (m["dim"] + m["rot_dim"]), m["q_rank"]), q + "dkv": (R + m["rot_dim"], W),
                    q + "dkv.norm": (R,), q + "uk": (H * m["dim"], R), q + "uv": (H * m["vdim"], R), q + "sink": (H,), q + "g": (H, W), q + "o": (W, H * m["vdim"])})
    else:
        a, C = m["left"], m["right"]["width"]
        H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
        out.update({q + "left.q": (H * D, W), q + "left.k": (G * D, W), q + "left.v": (G * V, W), q + "left.g": (H, W), q + "left.o": (W, H * V), q + "right.z": (C, W),
                    q + "right.z.b": (C,), q + "right.x": (C, W), q + "right.x.b": (C,), q + "right.g": (C, W), q + "right.o": (W, C), q + "left.out": (W,), q + "right.out": (W,)})
    if f:
        n = f["expert"]["ff"]
        out.update({p + "rg2": (W, W), p + "rg2.b": (W,), p + "mlp.router": (f["router"]["experts"], W)})
        for e in range(f["router"]["experts"]):
            out.update({p + f"mlp.e{e}.up": (n, W), p + f"mlp.e{e}.down": (W, n)})
    return out


def gated_weight(rng, name, shape):
    """A random tensor of a design whose sublayers join through gates: heads that mostly keep their own score, taps of one size, sinks that take
    a visible share."""
    a = rng.standard_normal(shape).astype(np.float32)
    leaf = name.split(".", 1)[1] if name[0] == "l" and name[1].isdigit() else name
    if leaf.endswith((".norm", "norm1", ".out")):
        a = 1 + 0.2 * a
    elif leaf.endswith(".talk"):
        a = 0.6 * np.eye(shape[0]) + a / np.sqrt(shape[0])
    elif leaf.endswith(".sink"):
        a += 1
    elif leaf.endswith(".b"):
        a *= 0.4
    elif leaf != "embed":
        a /= np.sqrt(shape[-1])
    return bf16_round(np.asarray(a, np.float32))[1]


def layered_shapes(cfg):
    """Tensor name -> shape of every tensor a configuration asks for."""
    W, out = cfg["width"], {"embed": (cfg["vocab"], cfg["width"])}
    for i, layer in enumerate(cfg["layers"]):
        if "streams" in cfg:
            out.update(streams_layer_shapes(layer, W, cfg["streams"], f"l{i}."))
            continue
        if cfg["architecture"] == "Zevilorn":
            out.update(gated_layer_shapes(layer, W, f"l{i}."))
            continue
        if layer.get("weights_of") is not None:
            continue
        if layer["type"].startswith("latent"):
            out.update(latent_layer_shapes(layer, W, f"l{i}."))
            continue
        m, p = layer["mixer"], f"l{i}."
        q, k, v = m["heads"] * m["dim"], m["kv_heads"] * m["dim"], m["kv_heads"] * m["vdim"]
        out.update({p + "norm1": (W,), p + "norm1b": (W,), p + "mix.q": (q, W), p + "mix.k": (k, W), p + "mix.v": (v, W), p + "mix.q.norm": (q,),
                    p + "mix.k.norm": (k,), p + "mix.g": (m["heads"], W), p + "mix.o": (W, m["heads"] * m["vdim"])})
        if layer["mlp"] is not None:
            f = layer["mlp"]["ff"]
            out.update({p + "norm2": (W,), p + "norm2b": (W,), p + "mlp.gate": (f, W), p + "mlp.up": (f, W), p + "mlp.down": (W, f)})
    out.update({"final.norm": (W,), "head": (cfg["vocab"], W)})
    return out


def layered_weights(rng, cfg):
    """Random bf16-exact fp32 weights: products of unit inputs have unit size, norms lie around 1."""
    w = {}
    for name, shape in layered_shapes(cfg).items():
        if "streams" in cfg:
            w[name] = streams_weight(rng, name, shape)
            continue
        if cfg["architecture"] == "Zevilorn":
            w[name] = gated_weight(rng, name, shape)
            continue
        a = rng.standard_normal(shape, dtype=np.float32)
        if name.endswith("mlp.act"):
            w[name] = bf16_round(0.6 * a)[1]
            continue
        w[name] = bf16_round(1.0 + 0.2 * a if len(shape) == 1 else (a if name == "embed" else a / np.sqrt(shape[1])))[1]
    return w


def write_layered(folder, cfg, weights, alias_layers=False):
    """Writes config.json and model.safetensors (bf16). `weights`: name -> fp32 array, or a function (name, shape)
    giving one. alias_layers: every layer's tensors (and every expert's) point at the bytes of the first one with that tensor and shape."""
    import json
    import re
    from pathlib import Path
    folder = Path(folder)
    folder.mkdir(parents=True, exist_ok=True)
    (folder / "config.json").write_text(json.dumps(cfg))
    header, stored, placed, off = {}, [], {}, 0
    for name, shape in layered_shapes(cfg).items():
        n = 2 * int(np.prod(shape))
        key = (re.sub(r"\.e\d+\.", ".e.", name.split(".", 1)[1]) if name[0] == "l" and name[1].isdigit() else name, shape)
        at = placed.get(key) if alias_layers else None
        if at is None:
            at = placed[key] = off
            stored.append((name, shape))
            off += n
        header[name] = {"dtype": "BF16", "shape": list(shape), "data_offsets": [at, at + n]}
    text = json.dumps(header).encode()
    text += b" " * ((-len(text)) % 8)
    with open(folder / "model.safetensors", "wb") as f:
        f.write(len(text).to_bytes(8, "little") + text)
        for name, shape in stored:
            a = weights(name, shape) if callable(weights) else weights[name]
            f.write(bf16_round(a)[0].tobytes())
