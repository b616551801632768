"""Plain, slow NumPy implementation of the decoder design "Gunuvik" (windowed grouped-query attention with a learned distance bias
and a sink, matrix-memory recurrence, sandwich norms), one function per mechanism.  Test infrastructure: it shares no code with the
product path.  Everything is computed in float64 over one whole sequence; there is no cache, so a sequence is run from its first
token every time.
"""
import math

import numpy as np


def _f(a):
    return np.asarray(a, dtype=np.float64)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def log_sigmoid(z):
    return -np.logaddexp(0.0, -z)


def rms(x, eps):
    """x / sqrt(mean x^2 + eps) over the last axis."""
    x = _f(x)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def linear(h, w, b=None):
    """w is [out, in]."""
    y = _f(h) @ _f(w).T
    return y if b is None else y + _f(b)


def distance_bucket(n, rows, far):
    """Row of a distance bias table with `rows` rows: the first half counts single distances, the second half is logarithmic up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(S, table, far):
    """[H, S, S]: entry (h, i, j) for i >= j (zero above the diagonal)."""
    table = _f(table)
    per = np.stack([table[distance_bucket(n, table.shape[0], far)] for n in range(S)])     # [S, H]
    out = np.zeros((table.shape[1], S, S))
    for i in range(S):
        out[:, i, :i + 1] = per[i - np.arange(i + 1)].T
    return out


def window_mask(S, size, keep_first):
    """True where position i sees position j."""
    i, j = np.arange(S)[:, None], np.arange(S)[None]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_with_sink(z, sink):
    """Weights of the scores z [.., keys] (-inf: not seen) when exp(sink) joins the denominator."""
    m = np.maximum(z.max(axis=-1, keepdims=True), sink)
    e = np.exp(z - m)
    return e / (e.sum(axis=-1, keepdims=True) + np.exp(sink - m))


def attention_keys(h, m, w, eps):
    """(normed keys [S, G, dim], values [S, G, vdim])."""
    S, G = h.shape[0], m["kv_heads"]
    k = linear(h, w["k"], w["k.b"]).reshape(S, G, m["dim"])
    v = linear(h, w["v"], w["v.b"]).reshape(S, G, m["vdim"])
    return rms(k, eps) * _f(w["k.norm"]), v


def attention(h, m, w, k, v, eps):
    """m: the layer's mixer sizes; w: its tensors; (k, v): the keys and values it attends to."""
    S, H, G, dim = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rms(linear(h, w["q"], w["q.b"]).reshape(S, H, dim), eps) * _f(w["q.norm"])
    bias = distance_bias(S, w["rel"], m["bias_max"])
    mask = window_mask(S, m["mask"]["size"], m["mask"]["keep_first"])
    gate = sigmoid(linear(h, w["g"]))
    out = np.zeros((S, H, m["vdim"]))
    for a in range(H):
        g = a // (H // G)
        z = np.where(mask, q[:, a] @ k[:, g].T * m["scale"] + bias[a], -np.inf)
        out[:, a] = softmax_with_sink(z, float(_f(w["sink"])[a])) @ v[:, g] * gate[:, a:a + 1]
    return linear(out.reshape(S, -1), w["o"])


def matrix_memory(q, k, v, i, f):
    """One head, token by token: q, k [S, dim], v [S, vdim], log gates i, f [S] -> [S, vdim]."""
    S, dim, vdim = q.shape[0], q.shape[1], v.shape[1]
    mem, n, m = np.zeros((dim, vdim)), np.zeros(dim), 0.0
    out = np.zeros((S, vdim))
    for t in range(S):
        new = max(f[t] + m, i[t])
        keep, add = math.exp(f[t] + m - new), math.exp(i[t] - new)
        mem = keep * mem + add * np.outer(k[t], v[t])
        n = keep * n + add * k[t]
        m = new
        out[t] = mem.T @ q[t] / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(h, m, w, eps):
    S, H, dim, vdim, cap = h.shape[0], m["heads"], m["dim"], m["vdim"], m["gate_cap"]
    q = linear(h, w["q"]).reshape(S, H, dim) * dim ** -0.5
    k = linear(h, w["k"]).reshape(S, H, dim)
    v = linear(h, w["v"]).reshape(S, H, vdim)
    i = cap * np.tanh(linear(h, w["i"], w["i.b"]) / cap)
    f = log_sigmoid(cap * np.tanh(linear(h, w["f"], w["f.b"]) / cap))
    o = np.stack([rms(matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a]), eps) for a in range(H)], axis=1).reshape(S, H * vdim)
    return linear(o * _f(w["norm"]) * sigmoid(linear(h, w["g"])), w["o"])


def gated_ff(h, w):
    z = linear(h, w["gate"])
    return linear(z * sigmoid(z) * linear(h, w["up"]), w["down"])


class GunuvikOracle:
    """cfg: the parsed config.json; weights: tensor name -> array."""

    def __init__(self, cfg, weights):
        self.cfg, self.w = cfg, weights

    def _part(self, p):
        return {k[len(p):]: v for k, v in self.w.items() if k.startswith(p)}

    def forward(self, ids, record=None):
        """ids [S] -> logits [S, vocab].  `record` (a list) receives the residual stream after every layer."""
        cfg, w = self.cfg, self.w
        eps = cfg["norm"]["eps"]
        x = _f(w["embed"])[np.asarray(ids)] * cfg["embedding"]["scale"]
        kept = {}
        for i, layer in enumerate(cfg["layers"]):
            l, m = "l%d." % i, layer["mixer"]
            h = rms(x, eps) * _f(w[l + "norm1"])
            mw = self._part(l + "mix.")
            if layer["type"] == "attention":
                src = m.get("kv_from")
                if src is None:
                    kept[i] = attention_keys(h, m, mw, eps)
                    src = i
                y = attention(h, m, mw, *kept[src], eps)
            else:
                y = mlstm(h, m, mw, eps)
            x = x + rms(y, eps) * _f(w[l + "norm1b"]) * _f(w[l + "ls1"])
            if layer["mlp"] is not None:
                y = gated_ff(rms(x, eps) * _f(w[l + "norm2"]), self._part(l + "mlp."))
                x = x + rms(y, eps) * _f(w[l + "norm2b"]) * _f(w[l + "ls2"])
            if record is not None:
                record.append(x.copy())
        return linear(rms(x, eps) * _f(w["final.norm"]), w["head"])
