"""Plain, slow NumPy implementation of the decoder design "Pepilix" (latent attention, short input convolutions, gated
parallel residual, experts chosen by token id), one function per mechanism.  Test infrastructure: it shares no code with the
product path.  Everything is computed in float64 over one whole sequence; there is no cache, so a sequence is run from its
first token every time.
"""
import numpy as np


def _f(a):
    return np.asarray(a, dtype=np.float64)


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * z))


def rms(x, w, eps):
    """x / sqrt(mean x^2 + eps) * w over the last axis."""
    x = _f(x)
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * _f(w)


def group_rms(x, w, groups, eps):
    """The vector is cut into `groups` equal parts, each normed by its own root mean square; one weight over the whole."""
    x = _f(x)
    parts = x.reshape(x.shape[:-1] + (groups, x.shape[-1] // groups))
    n = parts / np.sqrt(np.mean(parts * parts, axis=-1, keepdims=True) + eps)
    return n.reshape(x.shape) * _f(w)


def short_conv(h, w):
    """h [S, d], w [d, taps]: out[t] = sum_j w[:, j] h[t - taps + 1 + j], zeros before the start."""
    h, w = _f(h), _f(w)
    S, taps = h.shape[0], w.shape[1]
    out = np.zeros_like(h)
    for t in range(S):
        for j in range(taps):
            p = t - taps + 1 + j
            if p >= 0:
                out[t] += w[:, j] * h[p]
    return out


def rotate_half(x, positions, dims, base):
    """x [S, ..., n]: pairs (i, i + dims / 2) of the first `dims` values turn by position * base^(-2 i / dims)."""
    x = _f(x).copy()
    half = dims // 2
    for s, p in enumerate(positions):
        for i in range(half):
            a = float(p) * float(base) ** (-2.0 * i / dims)
            u, v = x[s, ..., i].copy(), x[s, ..., i + half].copy()
            x[s, ..., i] = u * np.cos(a) - v * np.sin(a)
            x[s, ..., i + half] = v * np.cos(a) + u * np.sin(a)
    return x


def latent_keys(h, w_dkv, norm_w, kv_rank, rot_dims, base, eps):
    """(latent c [S, kv_rank], rotated shared key part [S, rot_dim]) of every position."""
    d = _f(h) @ _f(w_dkv).T
    c = rms(d[:, :kv_rank], norm_w, eps)
    return c, rotate_half(d[:, kv_rank:], range(d.shape[0]), rot_dims, base)


def softmax(z):
    e = np.exp(z - z.max(axis=-1, keepdims=True))
    return e / e.sum(axis=-1, keepdims=True)


def latent_attention(h, m, w, c, kr):
    """m: the layer's mixer sizes; w: q, uk, uv, o; (c, kr): the latent and rotated key part the layer attends to."""
    S, H, dim, rot, vdim = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    q = (_f(h) @ _f(w["q"]).T).reshape(S, H, dim + rot)
    qn, qr = q[..., :dim], rotate_half(q[..., dim:], range(S), m["rot"]["dims"], m["rot"]["base"])
    k = (c @ _f(w["uk"]).T).reshape(S, H, dim)
    v = (c @ _f(w["uv"]).T).reshape(S, H, vdim)
    out = np.zeros((S, H, vdim))
    for a in range(H):
        z = (qn[:, a] @ k[:, a].T + qr[:, a] @ kr.T) * m["scale"]
        z = np.where(np.tril(np.ones((S, S), dtype=bool)), z, -np.inf)
        out[:, a] = softmax(z) @ v[:, a]
    return out.reshape(S, H * vdim) @ _f(w["o"]).T


def clamped_expert(h, gate, up, down, limit):
    g = np.minimum(_f(h) @ _f(gate).T, limit)
    u = np.clip(_f(h) @ _f(up).T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1.0)) @ _f(down).T


def table_experts(h, ids, table, experts, limit):
    """table [vocab, top] names the experts of every token id; each has weight 1 / top."""
    out = np.zeros((len(ids), experts[0]["down"].shape[0]))
    top = table.shape[1]
    for s, t in enumerate(ids):
        for e in table[int(t)]:
            x = experts[int(e)]
            out[s] += clamped_expert(h[s:s + 1], x["gate"], x["up"], x["down"], limit)[0] / top
    return out


class PepilixOracle:
    """cfg: the parsed config.json; weights: tensor name -> array."""

    def __init__(self, cfg, weights):
        self.cfg, self.w = cfg, weights

    def _mix(self, i):
        p = "l%d.mix." % i
        return {k[len(p):]: v for k, v in self.w.items() if k.startswith(p)}

    def _mlp(self, i):
        p, n = "l%d.mlp." % i, self.cfg["layers"][i]["mlp"]["router"]["experts"]
        ex = [{k: self.w["%se%d.%s" % (p, e, k)] for k in ("gate", "up", "down")} for e in range(n)]
        return np.asarray(self.w[p + "table"]), ex

    def forward(self, ids, record=None):
        """ids [S] -> logits [S, vocab].  `record` (a list) receives the residual stream after every layer."""
        cfg, w = self.cfg, self.w
        eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
        x = _f(w["embed"])[np.asarray(ids)] * cfg["embedding"]["scale"]
        kept = {}
        for i, layer in enumerate(cfg["layers"]):
            l, m = "l%d." % i, layer["mixer"]
            h1 = group_rms(x, w[l + "norm1"], groups, eps)
            hc = h1 + short_conv(h1, w[l + "canon1"])
            mw = self._mix(i)
            src = m.get("kv_from")
            if src is None:
                kept[i] = latent_keys(hc, mw["dkv"], mw["dkv.norm"], m["kv_rank"], m["rot"]["dims"], m["rot"]["base"], eps)
                src = i
            add = latent_attention(hc, m, mw, *kept[src]) * sigmoid(h1 @ _f(w[l + "rg1"]).T + _f(w[l + "rg1.b"]))
            if layer["mlp"] is not None:
                h2 = group_rms(x, w[l + "norm2"], groups, eps)
                table, ex = self._mlp(i)
                add = add + table_experts(h2, ids, table, ex, layer["mlp"]["expert"]["limit"]) * \
                    sigmoid(h2 @ _f(w[l + "rg2"]).T + _f(w[l + "rg2.b"]))
            x = x + add
            if record is not None:
                record.append(x.copy())
        return group_rms(x, w["final.norm"], groups, eps) @ _f(w["embed"]).T * cfg["logit_scale"]
