"""Plain, slow restatement of the layered language models in numpy, one function per mechanism. It
shares nothing with the product: the tests compare the library against it. `cfg` is a model's
config.json as a dict, `weights` maps tensor names to arrays, and everything runs in `dtype`
(float64 unless a test asks for something else)."""
import numpy as np


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z ** 3)))


def sinusoid(positions, width, dtype=np.float64):
    """[len(positions), width]: entry 2i = sin(p 10000^(-2i/width)), entry 2i+1 = the cosine."""
    p = np.asarray(positions, dtype)[:, None]
    n = np.arange(width)
    freq = (10000.0 ** (-(2.0 * (n // 2)) / width)).astype(dtype)
    ang = p * freq
    return np.where(n % 2 == 0, np.sin(ang), np.cos(ang)).astype(dtype)


def embed(tokens, positions, table, dtype=np.float64):
    return table[np.asarray(tokens)].astype(dtype) + sinusoid(positions, table.shape[1], dtype)


def query_temperature(positions, coef, every):
    p = np.asarray(positions)
    return 1.0 + coef * np.log(np.floor((p + 1) / every) + 1.0)


def alibi_slopes(heads):
    return np.array([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)])


def window_mask(q_pos, k_pos, size):
    """True where the key at k_pos is seen from q_pos: itself and the size - 1 tokens before it."""
    d = np.asarray(q_pos)[:, None] - np.asarray(k_pos)[None, :]
    return (d >= 0) & (d < size)


def distance_bias(scores, q_pos, k_pos, slope):
    return scores - slope * (np.asarray(q_pos)[:, None] - np.asarray(k_pos)[None, :])


def softmax_with_sink(scores, mask):
    """exp(s_j) / (1 + sum exp(s_j)) over the seen keys, evaluated around max(0, max s)."""
    s = np.where(mask, scores, -np.inf)
    m = np.maximum(s.max(axis=-1, keepdims=True), 0.0)
    e = np.where(mask, np.exp(s - m), 0.0)
    return e / (np.exp(-m) + e.sum(axis=-1, keepdims=True))


def head_gate(h, w_g):
    return 1.0 / (1.0 + np.exp(-(h @ w_g.T)))


def project_qkv(h, w, mixer, eps, positions):
    """Normed, temperature-scaled queries [T, H, dim], normed keys [T, G, dim] and values [T, G, vdim]."""
    T, H, G = len(h), mixer["heads"], mixer["kv_heads"]
    q = rms_norm(h @ w["q"].T, w["q.norm"], eps)
    k = rms_norm(h @ w["k"].T, w["k.norm"], eps)
    t = mixer.get("q_temp")
    if t:
        q = q * query_temperature(positions, t["coef"], t["every"])[:, None]
    return q.reshape(T, H, mixer["dim"]), k.reshape(T, G, mixer["dim"]), (h @ w["v"].T).reshape(T, G, mixer["vdim"])


def attend(q, k, v, q_pos, k_pos, mixer):
    """[Tq, H, vdim] of queries at q_pos over keys at k_pos."""
    H, G = mixer["heads"], mixer["kv_heads"]
    mask = window_mask(q_pos, k_pos, mixer["mask"]["size"])
    slopes = alibi_slopes(H)
    out = np.zeros((len(q_pos), H, v.shape[-1]), q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = distance_bias((q[:, h] @ k[:, g].T) * mixer["scale"], q_pos, k_pos, slopes[h])
        out[:, h] = softmax_with_sink(s, mask) @ v[:, g]
    return out


def attention(h, w, mixer, eps, positions, cache):
    """The mixer on new tokens; cache is a dict with 'k', 'v', 'pos' of earlier tokens (updated)."""
    q, k, v = project_qkv(h, w, mixer, eps, positions)
    if cache:
        k, v = np.concatenate([cache["k"], k]), np.concatenate([cache["v"], v])
        kp = np.concatenate([cache["pos"], positions])
    else:
        kp = np.asarray(positions)
    cache["k"], cache["v"], cache["pos"] = k, v, kp
    o = attend(q, k, v, positions, kp, mixer) * head_gate(h, w["g"])[:, :, None]
    return o.reshape(len(h), -1) @ w["o"].T


def feed_forward(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


class Model:
    """Runs a model whose layers attend through `attention` and whose feed-forwards are gated; a layer
    with 'weights_of' takes another layer's tensors and keeps a cache of its own."""

    def __init__(self, cfg, weights, dtype=np.float64):
        self.cfg, self.dtype = cfg, dtype
        self.w = {n: np.asarray(a, dtype) for n, a in weights.items()}

    def source(self, i):
        while self.cfg["layers"][i].get("weights_of") is not None:
            i = self.cfg["layers"][i]["weights_of"]
        return i

    def group(self, prefix):
        return {n[len(prefix):]: a for n, a in self.w.items() if n.startswith(prefix)}

    def new_state(self):
        return {"len": 0, "caches": [{} for _ in self.cfg["layers"]]}

    def forward(self, tokens, state=None, trace=None):
        """Logits [T, vocab] of the next tokens of a sequence; `trace` receives the residual after each layer."""
        state = self.new_state() if state is None else state
        eps = self.cfg["norm"]["eps"]
        pos = np.arange(state["len"], state["len"] + len(tokens))
        x = embed(tokens, pos, self.w["embed"], self.dtype)
        for i, layer in enumerate(self.cfg["layers"]):
            p = "l%d." % self.source(i)
            h = rms_norm(x, self.w[p + "norm1"], eps)
            m = attention(h, self.group(p + "mix."), layer["mixer"], eps, pos, state["caches"][i])
            x = x + rms_norm(m, self.w[p + "norm1b"], eps)
            if layer["mlp"] is not None:
                f = feed_forward(rms_norm(x, self.w[p + "norm2"], eps), self.group(p + "mlp."))
                x = x + rms_norm(f, self.w[p + "norm2b"], eps)
            if trace is not None:
                trace.append(x.copy())
        state["len"] += len(tokens)
        return rms_norm(x, self.w["final.norm"], eps) @ self.w["head"].T
