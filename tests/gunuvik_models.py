"""Small Gunuvik models for tests: configurations, seeded weights, a model folder on disk, and the oracle for them."""
import json
import os

import numpy as np

from oracle import gunuvik_oracle as GO
from oracle.gunuvik_oracle import GunuvikOracle
from seq2seqsharp_b200.gunuvik import config_from_json, engine_name, file_names
from seq2seqsharp_b200.safetensors_file import to_bfloat16, to_float32, write_safetensors
from tests.layered_models import rel, tokens  # noqa: F401  (re-exported)


def attention(heads, kv_heads, dim, vdim, window, keep, far=40, scale=None, kv_from=None, ff=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale or dim ** -0.5, "bias_max": far,
         "mask": {"size": window, "keep_first": keep}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def memory(heads, dim, vdim, cap=12.0, ff=None):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def config(layers, width, vocab, eps=1e-5, embed=1.0):
    return {"architecture": "Gunuvik", "embedding": {"scale": embed}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


CONFIGS = {
    # layers of unequal sizes, with and without a feed-forward, caches read by later layers through other windows
    "mixed": config([attention(6, 2, 16, 24, 20, 3, far=30, ff=40), attention(6, 2, 16, 24, 33, 5, far=25, scale=0.4, kv_from=0), memory(3, 16, 24, cap=9.0, ff=56),
                     attention(4, 4, 32, 16, 7, 0, ff=24), memory(2, 40, 8, cap=20.0), attention(4, 4, 32, 16, 12, 2, kv_from=3, ff=72)], 96, 101, embed=2.5),
    # nothing is a multiple of eight: no tensor-core path takes these shapes; more kept tokens than the window holds
    "odd": config([attention(3, 1, 10, 9, 4, 6, far=11, ff=13), memory(3, 7, 5, cap=3.0), attention(3, 1, 10, 9, 9, 1, far=50, kv_from=0, ff=9)], 50, 61, eps=1e-3, embed=3.0),
    # one head each, a window of one position
    "plain": config([attention(1, 1, 32, 32, 1, 2, ff=32), memory(1, 16, 16)], 64, 73),
    # wide enough for every tensor-core kernel
    "wide": config([attention(8, 2, 64, 64, 100, 10, far=90, ff=192), memory(4, 64, 128, ff=64), attention(8, 2, 64, 64, 70, 17, far=200, kv_from=0), memory(2, 128, 64, cap=15.0),
                    attention(6, 2, 128, 96, 1000, 0, far=64, ff=96)], 256, 300, embed=4.0),
}
REL_ROWS = {"mixed": [8, 12, 0, 6, 0, 16], "odd": [5, 0, 7], "plain": [4, 0], "wide": [16, 0, 32, 0, 8]}


def rel_rows(cfg):
    for n, c in CONFIGS.items():
        if c is cfg:
            return REL_ROWS[n]
    return [16] * len(cfg["layers"])


def layered(cfg, dtype="float32", rows=None):
    rows = rows or rel_rows(cfg)
    return config_from_json(cfg, dtype, {"l%d.mix.rel" % i: (r, layer["mixer"]["heads"]) for i, (r, layer) in enumerate(zip(rows, cfg["layers"]))
                                         if layer["type"] == "attention"})


def weights(cfg, seed=1, rows=None):
    """Tensor name -> float32 values that bfloat16 holds exactly."""
    rng = np.random.default_rng(seed)
    c = layered(cfg, rows=rows)
    names = file_names(c)
    out = {}
    for engine, shape in c.weight_shapes().items():
        n = names[engine]
        part = n.split(".", 1)[-1]
        if "norm" in part:
            w = rng.uniform(0.5, 1.5, size=shape)
        elif part in ("ls1", "ls2"):
            w = rng.uniform(0.3, 1.2, size=shape)
        elif part == "mix.rel":
            w = rng.normal(0, 1.5, size=shape)
        elif part == "mix.sink":
            w = rng.normal(1.0, 1.0, size=shape)
        elif part == "mix.f.b":
            w = rng.uniform(-2.0, 7.0, size=shape)      # heads that forget at once and heads that keep for hundreds of tokens
        elif part.endswith(".b"):
            w = rng.normal(0, 0.7, size=shape)
        elif n == "embed":
            w = rng.normal(0, 1.0, size=shape)
        else:
            w = rng.normal(0, (2.0 if part in ("mix.g", "mix.i", "mix.f") else 1.0) / np.sqrt(shape[1]), size=shape)
        a = to_float32(to_bfloat16(w.astype(np.float32)))
        out[n] = a.reshape(-1) if is_vector(part) else a
    return out


def is_vector(part):   # stored with one dimension
    return "norm" in part or part in ("ls1", "ls2", "mix.sink") or part.endswith(".b")


def engine_weights(cfg, w, rows=None):
    c = layered(cfg, rows=rows)
    return {engine_name(k, c): to_bfloat16(v) for k, v in w.items()}


def save(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: to_bfloat16(v) for k, v in w.items()})
    return str(path)


def oracle(cfg, w):
    return GunuvikOracle(cfg, w)


def needle(at, n, window, keep, scale=1.0, seed=9, layers=1, dim=16, vdim=16, heads=4, kv_heads=2):
    """(configuration, weights, ids): one marker token whose key stands out for every query, so that the output hangs on whether it is seen.

    Component 0 of the residual is the same for every token and component 1 marks the marker; queries have a constant large first element,
    keys have one only at the marker."""
    cfg = config([attention(heads, kv_heads, dim, vdim, window, keep, far=60, scale=scale)] +
                 [attention(heads, kv_heads, dim, vdim, window, keep, far=60, scale=scale, kv_from=0) for _ in range(layers - 1)], 64, 50)
    w = weights(cfg, seed)
    ids = [t if t != 49 else 48 for t in tokens(cfg, n, at)]
    ids[at] = 49
    w["embed"][:, 1] = 0.0
    w["embed"][49, 1] = 24.0
    for i in range(layers):
        p = "l%d." % i
        w[p + "norm1"][1] = 1.0
        w[p + "mix.rel"] *= 0.1
        w[p + "mix.sink"][:] = 1.0
        w[p + "mix.q"] *= 0.25
        for h in range(heads):
            w[p + "mix.q.b"][h * dim] = 6.0
        w[p + "mix.q.norm"][0] = 1.0
    w["l0.mix.k.norm"][0] = 1.0
    for g in range(kv_heads):
        w["l0.mix.k"][g * dim] = 0.0
        w["l0.mix.k"][g * dim, 1] = 1.0
        w["l0.mix.k.b"][g * dim] = 0.0
    return cfg, {k: to_float32(to_bfloat16(v)) for k, v in w.items()}, ids


TOL = {"float32": 1e-5, "bfloat16": 4e-2}


def _rounded(a):
    return to_float32(to_bfloat16(np.asarray(a, dtype=np.float32))).astype(np.float64)


def sensitivity(cfg, w, ids, want, n=6):
    """How far bfloat16 rounding of what enters and leaves the matrix products moves the logits of each position, in units of their
    spread.  A head whose output is nearly zero before its norm (a key almost orthogonal to the query, everything else forgotten) makes
    a position many times more sensitive than its neighbours."""
    real, out = GO.linear, np.zeros(len(ids))
    for seed in range(n):
        rng = np.random.default_rng(seed)

        def linear(h, wt, b=None):
            y = real(_rounded(h), wt, b)
            return _rounded(y * (1.0 + 2.0 ** -10 * rng.uniform(-1, 1, size=y.shape)))
        GO.linear = linear
        try:
            out = np.maximum(out, np.sqrt(((oracle(cfg, w).forward(ids) - want) ** 2).mean(axis=-1)) / want.std())
        finally:
            GO.linear = real
    return out


class Expected:
    """Oracle logits of a text and the error that each position may have."""

    def __init__(self, cfg, w, ids, dtype):
        self.ids, self.want = list(ids), oracle(cfg, w).forward(ids)
        self.spread = self.want.std()
        s = sensitivity(cfg, w, ids, self.want)
        self.allow = np.maximum(TOL[dtype], 4.0 * s * (1.0 if dtype == "bfloat16" else 2.0 ** -12))

    def worst(self, got, at=None):
        """Largest error over the allowed one; `at`: the positions that `got` holds (default: all)."""
        at = np.arange(len(self.ids)) if at is None else np.atleast_1d(np.arange(len(self.ids))[at])
        err = np.sqrt(((np.asarray(got, np.float64) - self.want[at]) ** 2).mean(axis=-1)) / self.spread
        return float((err / self.allow[at]).max())
