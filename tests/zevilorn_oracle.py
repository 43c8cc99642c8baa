"""Plain, slow restatement of models whose sublayers share one norm and add their gated results side by side, whose layers may run
in a loop, and whose mixers are grouped attention over convolved projections with heads that mix their scores, attention over
latents with queries through a latent of their own, or windowed attention beside a minimal gated recurrence. numpy, one function
per mechanism. It shares nothing with the product: the tests compare the library against it. `cfg` is a model's config.json as
a dict, `weights` maps tensor names to arrays, and everything runs in `dtype` (float64 unless a test asks for something
else)."""
import math

import numpy as np

_erf = np.vectorize(math.erf, otypes=[np.float64])


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / np.sqrt(2.0)))


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


# ---- rotation ------------------------------------------------------------------------------------------------
def frequencies(rot):
    return np.array([rot["base"] ** (-2.0 * i / rot["dims"]) for i in range(rot["dims"] // 2)])


def scale_linear(f, s):
    return f / s["factor"]


def scale_banded(f, s):
    """Short wavelengths stay, long ones are stretched by the factor, and a ramp in original / wavelength lies between."""
    out = []
    for x in f:
        turns = s["original"] * x / (2.0 * math.pi)
        if turns > s["high"]:
            out.append(x)
        elif turns < s["low"]:
            out.append(x / s["factor"])
        else:
            t = (turns - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - t) * x / s["factor"] + t * x)
    return np.array(out)


def rotate_neighbours(x, pos, f):
    """x [T, heads, dim]: entries 2i and 2i + 1 of the first 2 len(f) turn by pos f_i."""
    a = np.asarray(pos)[:, None, None] * f
    n = 2 * len(f)
    u, v, out = x[..., 0:n:2], x[..., 1:n:2], x.copy()
    out[..., 0:n:2] = u * np.cos(a) - v * np.sin(a)
    out[..., 1:n:2] = v * np.cos(a) + u * np.sin(a)
    return out


def rotate_halves(x, pos, f):
    """The same for entries i and i + len(f)."""
    a = np.asarray(pos)[:, None, None] * f
    n = len(f)
    u, v, out = x[..., :n], x[..., n:2 * n], x.copy()
    out[..., :n] = u * np.cos(a) - v * np.sin(a)
    out[..., n:2 * n] = v * np.cos(a) + u * np.sin(a)
    return out


# ---- attention -----------------------------------------------------------------------------------------------
def causal(q_pos, k_pos):
    return np.asarray(k_pos)[None, :] <= np.asarray(q_pos)[:, None]


def window(q_pos, k_pos, size):
    d = np.asarray(q_pos)[:, None] - np.asarray(k_pos)[None, :]
    return (d >= 0) & (d < size)


def scores(q, k, scale):
    """q [Tq, H, dim], k [Tk, G, dim] -> [H, Tq, Tk]."""
    H, G = q.shape[1], k.shape[1]
    return np.stack([q[:, h] @ k[:, h // (H // G)].T * scale for h in range(H)])


def soft_cap(s, cap):
    return cap * np.tanh(s / cap)


def mix_heads(s, talk):
    """s [H, ..]: head h's scores become sum_g talk[h][g] s_g."""
    return np.tensordot(talk, s, 1)


def weights_over(s, mask, sink=None):
    """Softmax over the seen keys. sink [H]: scores of one more entry of the denominator per head."""
    s = np.where(mask, s, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        sink = np.asarray(sink)[:, None, None]
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(sink - m) if sink is not None else 0.0))


def weighted_values(p, v):
    """p [H, Tq, Tk], v [Tk, G, vdim] -> [Tq, H, vdim]."""
    H, G = len(p), v.shape[1]
    return np.stack([p[h] @ v[:, h // (H // G)] for h in range(H)], 1)


def causal_conv(u, taps, past):
    """u [T, C], taps [C, n] (the last column meets the current token), past [n - 1, C] -> (sums, new past)."""
    n = taps.shape[1]
    full = np.concatenate([past, u])
    return sum(full[j:j + len(u)] * taps[:, j] for j in range(n)), full[len(full) - (n - 1):]


def extend(cache, **new):
    for n, a in new.items():
        cache[n] = np.concatenate([cache[n], a]) if n in cache else np.asarray(a)


def talking_attention(h, w, m, pos, cache):
    T, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    x = {}
    for n, c in (("q", H * D), ("k", G * D), ("v", G * V)):
        past = cache.get("past_" + n, np.zeros((m["conv"] - 1, c), h.dtype))
        x[n], cache["past_" + n] = causal_conv(h @ w[n].T + w[n + ".b"], w[n + ".conv"], past)
    f = frequencies(m["rot"])
    if m["rot"].get("scaling"):
        f = scale_banded(f, m["rot"]["scaling"])
    q = rotate_neighbours(x["q"].reshape(T, H, D), pos, f)
    extend(cache, k=rotate_neighbours(x["k"].reshape(T, G, D), pos, f), v=x["v"].reshape(T, G, V), pos=np.asarray(pos))
    s = mix_heads(soft_cap(scores(q, cache["k"], m["scale"]), m["softcap"]), w["talk"])
    p = weights_over(s, window(pos, cache["pos"], m["mask"]["size"]), np.zeros(H))
    return weighted_values(p, cache["v"]).reshape(T, -1) @ w["o"].T + w["o.b"]


def latent_attention(h, w, m, eps, pos, cache):
    T, H, D, R, V, K = len(h), m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).reshape(T, H, D + R)
    kv = h @ w["dkv"].T
    f = frequencies(m["rot"])
    extend(cache, c=rms_norm(kv[:, :K], w["dkv.norm"], eps), r=rotate_halves(kv[:, None, K:], pos, f), pos=np.asarray(pos))
    n = len(cache["pos"])
    k = np.concatenate([(cache["c"] @ w["uk"].T).reshape(n, H, D), np.repeat(cache["r"], H, 1)], -1)
    q = np.concatenate([q[..., :D], rotate_halves(q[..., D:], pos, f)], -1)
    p = weights_over(scores(q, k, m["scale"]), causal(pos, cache["pos"]), w["sink"])
    o = weighted_values(p, (cache["c"] @ w["uv"].T).reshape(n, H, V)) * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, -1) @ w["o"].T


def windowed_attention(h, w, m, pos, cache):
    T, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    f = frequencies(m["rot"])
    if m["rot"].get("scaling"):
        f = scale_linear(f, m["rot"]["scaling"])
    q = rotate_neighbours((h @ w["q"].T).reshape(T, H, D), pos, f)
    extend(cache, k=rotate_neighbours((h @ w["k"].T).reshape(T, G, D), pos, f), v=(h @ w["v"].T).reshape(T, G, V), pos=np.asarray(pos))
    p = weights_over(scores(q, cache["k"], m["scale"]), window(pos, cache["pos"], m["mask"]["size"]))
    o = weighted_values(p, cache["v"]) * sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, -1) @ w["o"].T


# ---- recurrence ----------------------------------------------------------------------------------------------
def candidate(u):
    return np.where(u >= 0, u + 0.5, sigmoid(u))


def gated_scan(z, c, S):
    """Token by token S <- (1 - z) S + z c; all of S [T, width]."""
    out = np.zeros_like(c)
    for t in range(len(c)):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out[t] = S
    return out


def min_gru(h, w, state):
    z, c = sigmoid(h @ w["z"].T + w["z.b"]), candidate(h @ w["x"].T + w["x.b"])
    S = gated_scan(z, c, state.get("S", np.zeros(z.shape[1], h.dtype)))
    state["S"] = S[-1]
    return (S * silu(h @ w["g"].T)) @ w["o"].T


def normed_half_sum(a, b, wa, wb, eps):
    return 0.5 * (rms_norm(a, wa, eps) + rms_norm(b, wb, eps))


# ---- feed-forward --------------------------------------------------------------------------------------------
def best_groups(s, groups, keep):
    """s [T, n] with everything outside each row's best groups at minus infinity; a group counts by its two largest."""
    two = np.sort(s.reshape(len(s), groups, -1), -1)[..., -2:].sum(-1)
    order = np.argsort(-two, axis=-1, kind="stable")[:, :keep]
    open_ = np.zeros(two.shape, bool)
    np.put_along_axis(open_, order, True, axis=-1)
    return np.where(np.repeat(open_, s.shape[1] // groups, axis=1), s, -np.inf)


def route(h, w, r):
    """(ids [T, top], weights [T, top])."""
    s = sigmoid(h @ w["router"].T)
    choice = best_groups(s, r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else s
    ids = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    return ids, np.take_along_axis(s, ids, axis=-1)


def experts(h, w, mlp):
    r = mlp["router"]
    ids, p = route(h, w, r)
    out = np.zeros_like(h)
    for e in range(r["experts"]):
        rows, k = np.nonzero(ids == e)
        if len(rows):
            out[rows] += p[rows, k][:, None] * (gelu_erf(h[rows] @ w[f"e{e}.up"].T) @ w[f"e{e}.down"].T)
    return out


# ---- layers --------------------------------------------------------------------------------------------------
def residual_gate(h, w, b):
    return sigmoid(h @ w.T + b)


def runs(cfg):
    """[(layer, whether the embedding is added in front of it)] in the order in which layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    return [(i, False) for i in range(a)] + [(i, t > 0 and i == a) for t in range(loop["times"]) for i in range(a, b)] + [(i, False) for i in range(b, n)]


class Model:
    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.dtype = cfg, dtype
        self.w = {n: np.asarray(a, dtype) for n, a in weights.items()}

    def group(self, prefix):
        return {n[len(prefix):]: a for n, a in self.w.items() if n.startswith(prefix)}

    def new_state(self):
        return {"len": 0, "caches": [({}, {}) for _ in runs(self.cfg)]}

    def mixer(self, h, p, layer, pos, caches):
        m, eps = layer["mixer"], self.cfg["norm"]["eps"]
        if layer["type"] == "attention":
            return talking_attention(h, self.group(p + "mix."), m, pos, caches[0])
        if layer["type"] == "latent_attention":
            return latent_attention(h, self.group(p + "mix."), m, eps, pos, caches[0])
        return normed_half_sum(windowed_attention(h, self.group(p + "mix.left."), m["left"], pos, caches[0]),
                               min_gru(h, self.group(p + "mix.right."), caches[1]), self.w[p + "mix.left.out"], self.w[p + "mix.right.out"], eps)

    def forward(self, tokens, state=None, trace=None):
        """Logits [T, vocab] of the next tokens of a sequence; `trace` receives the residual after each layer run."""
        state = self.new_state() if state is None else state
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        pos = np.arange(state["len"], state["len"] + len(tokens))
        x = first = self.w["embed"][np.asarray(tokens)]
        for run, (i, again) in enumerate(runs(cfg)):
            layer, p = cfg["layers"][i], f"l{i}."
            if again:
                x = x + first
            h = rms_norm(x, self.w[p + "norm1"], eps)
            y = self.mixer(h, p, layer, pos, state["caches"][run]) * residual_gate(h, self.w[p + "rg1"], self.w[p + "rg1.b"])
            if layer["mlp"] is not None:
                y = y + experts(h, self.group(p + "mlp."), layer["mlp"]) * residual_gate(h, self.w[p + "rg2"], self.w[p + "rg2.b"])
            x = x + y
            if trace is not None:
                trace.append(x)
        state["len"] += len(tokens)
        return rms_norm(x, self.w["final.norm"], eps) @ self.w["head"].T
