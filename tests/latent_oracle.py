"""Plain, slow restatement of models with latent attention, polynomial feed-forwards and experts, in numpy, one
function per mechanism. It shares nothing with the product: the tests compare the library against it. `cfg` is a
model's config.json as a dict, `weights` maps tensor names to arrays, and everything runs in `dtype` (float64 unless a
test asks for something else)."""
import math

import numpy as np


def root_mean_square(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def rms_norm(x, w, eps):
    return x / root_mean_square(x, eps) * w


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


# ---- rotation ------------------------------------------------------------------------------------------------
def frequencies(rot):
    """(frequency of each pair, factor on cosine and sine)."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = np.array([base ** (-2.0 * i / n) for i in range(n // 2)])
    if not s:
        return f, 1.0
    turns = lambda t: n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    lo, hi = max(math.floor(turns(s["fast"])), 0), min(math.ceil(turns(s["slow"])), n - 1)
    ramp = np.clip((np.arange(n // 2) - lo) / max(hi - lo, 0.001), 0, 1)
    return f / s["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, positions, rot):
    """x [T, .., dims]: entry i turns with entry i + dims / 2."""
    f, mul = frequencies(rot)
    a = np.asarray(positions, x.dtype).reshape(-1, *[1] * (x.ndim - 1)) * f.astype(x.dtype)
    c, s = np.cos(a) * mul, np.sin(a) * mul
    u, v = np.split(x, 2, axis=-1)
    return np.concatenate([u * c - v * s, v * c + u * s], axis=-1)


# ---- attention -----------------------------------------------------------------------------------------------
def visible(q_pos, k_pos, window):
    """True where the key is seen: not later, and (window given) at most window - 1 tokens back."""
    d = np.asarray(q_pos)[:, None] - np.asarray(k_pos)[None, :]
    return (d >= 0) & (d < window) if window else d >= 0


def softmax(scores, mask=None):
    s = scores if mask is None else np.where(mask, scores, -np.inf)
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latents(h, w, mixer, eps, positions):
    """What a token leaves in the cache: the normed latent and the rotated key part that all heads share."""
    y = h @ w["dkv"].T
    r = mixer["kv_rank"]
    return rms_norm(y[:, :r], w["dkv.norm"], eps), rotate(y[:, r:], positions, mixer["rot"])


def queries(h, w, mixer, positions):
    q = (h @ w["q"].T).reshape(len(h), mixer["heads"], mixer["dim"] + mixer["rot_dim"])
    return q[:, :, :mixer["dim"]], rotate(q[:, :, mixer["dim"]:], positions, mixer["rot"])


def attend(q, q_rot, c, k_rot, w, mixer, q_pos, k_pos):
    """[Tq, heads, vdim]: every head makes its keys and values from the latents."""
    H, D, V = mixer["heads"], mixer["dim"], mixer["vdim"]
    mask = visible(q_pos, k_pos, (mixer.get("mask") or {}).get("size"))
    out = np.zeros((len(q_pos), H, V), q.dtype)
    for h in range(H):
        k, v = c @ w["uk"][h * D:(h + 1) * D].T, c @ w["uv"][h * V:(h + 1) * V].T
        out[:, h] = softmax((q[:, h] @ k.T + q_rot[:, h] @ k_rot.T) * mixer["scale"], mask) @ v
    return out


def latent_attention(h, w, mixer, eps, positions, cache, gated):
    """The mixer on new tokens. cache: a dict of earlier tokens' 'c', 'r', 'pos', extended here unless the layer reads
    another layer's (then that layer has done so already)."""
    if mixer.get("kv_from") is None:
        c, r = latents(h, w, mixer, eps, positions)
        for n, a in (("c", c), ("r", r), ("pos", np.asarray(positions))):
            cache[n] = np.concatenate([cache[n], a]) if n in cache else a
    q, qr = queries(h, w, mixer, positions)
    o = attend(q, qr, cache["c"], cache["r"], w, mixer, positions, cache["pos"]).reshape(len(h), -1)
    if gated:
        o = o * sigmoid(h @ w["g"].T)
    return o @ w["o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------
def poly_norm(z, coef, eps):
    a, b, c, e = coef
    n = lambda v: v / root_mean_square(v, eps)
    return a * n(z) + b * n(z * z) + c * n(z * z * z) + e


def dense(h, w, eps):
    return poly_norm(h @ w["up"].T, w["act"], eps) @ w["down"].T


def route(h, w_router, top):
    """(chosen experts [T, top], their scores)."""
    s = softmax(h @ w_router.T)
    ids = np.argsort(-s, axis=-1, kind="stable")[:, :top]
    return ids, np.take_along_axis(s, ids, axis=-1)


def clamped_glu(g, u, limit):
    g, u = np.minimum(g, limit), np.clip(u, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1)


def expert(h, w, prefix, limit):
    return clamped_glu(h @ w[prefix + "gate"].T, h @ w[prefix + "up"].T, limit) @ w[prefix + "down"].T


def experts(h, w, mlp):
    ids, weight = route(h, w["router"], mlp["router"]["top"])
    out = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        rows, k = np.nonzero(ids == e)
        if len(rows):
            out[rows] += weight[rows, k][:, None] * expert(h[rows], w, f"e{e}.", mlp["expert"]["limit"])
    return out


# ---- model ---------------------------------------------------------------------------------------------------
class Model:
    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.dtype = cfg, dtype
        self.w = {n: np.asarray(a, dtype) for n, a in weights.items()}

    def group(self, prefix):
        return {n[len(prefix):]: a for n, a in self.w.items() if n.startswith(prefix)}

    def new_state(self):
        return {"len": 0, "caches": [{} for _ in self.cfg["layers"]]}

    def forward(self, tokens, state=None, trace=None):
        """Logits [T, vocab] of the next tokens of a sequence; `trace` receives the residual after each layer."""
        state = self.new_state() if state is None else state
        eps = self.cfg["norm"]["eps"]
        pos = np.arange(state["len"], state["len"] + len(tokens))
        x = self.w["embed"][np.asarray(tokens)]
        for i, layer in enumerate(self.cfg["layers"]):
            p, m = f"l{i}.", layer["mixer"]
            cache = state["caches"][i if m.get("kv_from") is None else m["kv_from"]]
            y = latent_attention(x, self.group(p + "mix."), m, eps, pos, cache, layer["type"] == "latent_attention_2")
            x = x + rms_norm(y, self.w[p + "norm1"], eps)
            mlp = layer["mlp"]
            if mlp is not None:
                w = self.group(p + "mlp.")
                f = dense(x, w, eps) if mlp["kind"] == "dense" else experts(x, w, mlp)
                x = x + rms_norm(f, self.w[p + "norm2"], eps)
            if trace is not None:
                trace.append(x.copy())
        state["len"] += len(tokens)
        return rms_norm(x, self.w["final.norm"], eps) @ self.w["head"].T
