"""Plain, slow restatement of models whose mixers are grouped attention with kept first tokens, or chunked attention beside
a gated delta rule; whose residual is several streams; and whose experts are picked within groups. numpy, one function per
mechanism. It shares nothing with the product: the tests compare the library against it. `cfg` is a model's config.json as
a dict, `weights` maps tensor names to arrays, and everything runs in `dtype` (float64 unless a test asks for something
else)."""
import numpy as np


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def rms(x, eps):
    return np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def shifted_norm(x, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return x / rms(x, eps) * (1.0 + w)


def softmax(s):
    e = np.exp(s - s.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


# ---- which keys are seen -------------------------------------------------------------------------------------
def window_with_kept(q_pos, k_pos, size, keep):
    q, k = np.asarray(q_pos)[:, None], np.asarray(k_pos)[None, :]
    return (k <= q) & ((q - k < size) | (k < keep))


def same_chunk(q_pos, k_pos, size):
    q, k = np.asarray(q_pos)[:, None], np.asarray(k_pos)[None, :]
    return (k <= q) & (k // size == q // size)


# ---- attention -----------------------------------------------------------------------------------------------
def slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def weights_over(scores, mask, sink=None):
    """Softmax over the seen keys; a sink is one more entry of the denominator."""
    s = np.where(mask, scores, -np.inf)
    m = s.max(axis=-1, keepdims=True)
    if sink is not None:
        m = np.maximum(m, sink)
    e = np.exp(s - m)
    return e / (e.sum(axis=-1, keepdims=True) + (np.exp(sink - m) if sink is not None else 0.0))


def grouped_attention(q, k, v, mask, scale, slope=None, dist=None, sink=None):
    """q [Tq, H, dim], k [Tk, G, dim], v [Tk, G, vdim] -> [Tq, H, vdim]."""
    H, G = q.shape[1], k.shape[1]
    out = np.zeros((len(q), H, v.shape[-1]), q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if slope is not None:
            s = s - slope[h] * dist
        out[:, h] = weights_over(s, mask, None if sink is None else sink[h]) @ v[:, g]
    return out


def extend(cache, **new):
    for n, a in new.items():
        cache[n] = np.concatenate([cache[n], a]) if n in cache else np.asarray(a)


def kept_window_attention(h, w, m, eps, pos, cache):
    """Keys double as values (as projected); queries and keys are normed per head; the distance is taken off the score."""
    T, H, G, D = len(h), m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, D)
    raw = (h @ w["k"].T + w["k.b"]).reshape(T, G, D)
    extend(cache, k=raw / rms(raw, eps) * w["k.norm"], v=raw, pos=np.asarray(pos))
    q = q / rms(q, eps) * w["q.norm"]
    mask = window_with_kept(pos, cache["pos"], m["mask"]["size"], m["mask"]["keep_first"])
    dist = np.asarray(pos)[:, None] - cache["pos"][None, :]
    o = grouped_attention(q, cache["k"], cache["v"], mask, m["scale"], slopes(H), dist)
    return o.reshape(T, -1) @ w["o"].T + w["o.b"]


def chunked_attention(h, w, m, pos, cache):
    T, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).reshape(T, H, D)
    extend(cache, k=(h @ w["k"].T + w["k.b"]).reshape(T, G, D), v=(h @ w["v"].T + w["v.b"]).reshape(T, G, V), pos=np.asarray(pos))
    mask = same_chunk(pos, cache["pos"], m["mask"]["size"])
    return grouped_attention(q, cache["k"], cache["v"], mask, m["scale"], sink=w["sink"]).reshape(T, -1) @ w["o"].T


# ---- gated delta rule ----------------------------------------------------------------------------------------
def causal_conv(x, taps, past):
    """x [T, C], taps [C, n] (the last column meets the current token), past [n - 1, C] -> (silu of the sums, new past)."""
    n = taps.shape[1]
    full = np.concatenate([past, x])
    y = sum(full[j:j + len(x)] * taps[:, j] for j in range(n))
    return silu(y), full[len(full) - (n - 1):]


def unit(x):
    return x / np.sqrt((x * x).sum(-1, keepdims=True) + 1e-6)


def decays(h, w, heads, dim):
    """[T, heads, dim] factors in (0, 1)."""
    z = (h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]
    return np.exp(-np.exp(w["A_log"])[:, None] * softplus(z).reshape(len(h), heads, dim))


def delta_rule(q, k, v, g, beta, S):
    """One head, token by token. q, k, g [T, dim], v [T, vdim], beta [T], S [dim, vdim] (changed in place)."""
    o = np.zeros_like(v)
    for t in range(len(q)):
        S *= g[t][:, None]
        u = beta[t] * (v[t] - S.T @ k[t])
        S += np.outer(k[t], u)
        o[t] = S.T @ q[t]
    return o


def gated_delta(h, w, m, eps, state):
    T, H, G, D, V = len(h), m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    if not state:
        state["S"] = np.zeros((H, D, V), h.dtype)
        for n, c in (("q", G * D), ("k", G * D), ("v", H * V)):
            state[n] = np.zeros((m["conv"] - 1, c), h.dtype)
    x = {}
    for n in "qkv":
        x[n], state[n] = causal_conv(h @ w[n].T, w[n + ".conv"], state[n])
    q, k, v = unit(x["q"].reshape(T, G, D)) * D ** -0.5, unit(x["k"].reshape(T, G, D)), x["v"].reshape(T, H, V)
    g, beta = decays(h, w, H, D), sigmoid(h @ w["b"].T)
    o = np.stack([delta_rule(q[:, i // (H // G)], k[:, i // (H // G)], v[:, i], g[:, i], beta[:, i], state["S"][i]) for i in range(H)], 1)
    o = o / rms(o, eps) * w["norm"] * sigmoid((h @ w["g1"].T) @ w["g2"].T).reshape(T, H, V)
    return o.reshape(T, -1) @ w["o"].T


# ---- feed-forward --------------------------------------------------------------------------------------------
def gated_ff(h, w, prefix=""):
    return (silu(h @ w[prefix + "gate"].T) * (h @ w[prefix + "up"].T)) @ w[prefix + "down"].T


def best_groups(choice, groups, keep):
    """choice [T, n] with everything outside each row's best groups at minus infinity."""
    best = choice.reshape(len(choice), groups, -1).max(-1)
    order = np.argsort(-best, axis=-1, kind="stable")[:, :keep]
    open_ = np.zeros(best.shape, bool)
    np.put_along_axis(open_, order, True, axis=-1)
    return np.where(np.repeat(open_, choice.shape[1] // groups, axis=1), choice, -np.inf)


def route(h, w, r):
    """(ids [T, top], weights [T, top]); ids from r['experts'] on are identity experts."""
    s = softmax(h @ w["router"].T)
    choice = best_groups(s + w["correction"], r["groups"]["count"], r["groups"]["keep"])
    ids = np.argsort(-choice, axis=-1, kind="stable")[:, :r["top"]]
    p = np.take_along_axis(s, ids, axis=-1)
    return ids, p / (p.sum(-1, keepdims=True) + 1e-20) * r["scale"]


def experts(h, w, mlp):
    r = mlp["router"]
    ids, p = route(h, w, r)
    out = h * np.where(ids >= r["experts"], p, 0.0).sum(-1, keepdims=True)
    for e in range(r["experts"]):
        rows, k = np.nonzero(ids == e)
        if len(rows):
            out[rows] += p[rows, k][:, None] * gated_ff(h[rows], w, f"e{e}.")
    return out + gated_ff(h, w, "shared.")


# ---- streams -------------------------------------------------------------------------------------------------
def read_streams(x, w_in):
    """x [streams, T, width] -> what a sublayer reads."""
    return np.tensordot(w_in, x, 1)


def write_streams(x, mix, w_out, y):
    """mix [from, to]."""
    return np.tensordot(mix.T, x, 1) + w_out[:, None, None] * y


# ---- model ---------------------------------------------------------------------------------------------------
class Model:
    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.dtype = cfg, dtype
        self.w = {n: np.asarray(a, dtype) for n, a in weights.items()}

    def group(self, prefix):
        return {n[len(prefix):]: a for n, a in self.w.items() if n.startswith(prefix)}

    def new_state(self):
        return {"len": 0, "caches": [({}, {}) for _ in self.cfg["layers"]]}

    def mixer(self, h, p, layer, pos, caches):
        m, eps = layer["mixer"], self.cfg["norm"]["eps"]
        if layer["type"] == "attention":
            return kept_window_attention(h, self.group(p + "mix."), m, eps, pos, caches[0])
        return m["left_scale"] * chunked_attention(h, self.group(p + "mix.left."), m["left"], pos, caches[0]) + \
            m["right_scale"] * gated_delta(h, self.group(p + "mix.right."), m["right"], eps, caches[1])

    def forward(self, tokens, state=None, trace=None):
        """Logits [T, vocab] of the next tokens of a sequence; `trace` receives the sum of the streams after each layer."""
        state = self.new_state() if state is None else state
        cfg, eps = self.cfg, self.cfg["norm"]["eps"]
        pos = np.arange(state["len"], state["len"] + len(tokens))
        x = np.stack([self.w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]] * cfg["streams"])
        for i, layer in enumerate(cfg["layers"]):
            p = f"l{i}."
            for q in (1, 2):
                if q == 2 and layer["mlp"] is None:
                    continue
                hc = self.group(f"{p}hc{q}.")
                h = shifted_norm(read_streams(x, hc["in"]), self.w[f"{p}norm{q}"], eps)
                if q == 1:
                    y = self.mixer(h, p, layer, pos, state["caches"][i])
                else:
                    y = (gated_ff if layer["mlp"]["kind"] == "dense" else experts)(h, self.group(p + "mlp."), *([] if layer["mlp"]["kind"] == "dense" else [layer["mlp"]]))
                x = write_streams(x, hc["mix"], hc["out"], y)
            if trace is not None:
                trace.append(x.sum(0))
        state["len"] += len(tokens)
        z = shifted_norm(x.sum(0), self.w["final.norm"], eps) @ self.w["head"].T
        return cfg["logit_softcap"] * np.tanh(z / cfg["logit_softcap"])
