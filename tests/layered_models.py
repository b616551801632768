"""Small Pepilix models for tests: configurations, seeded weights, a model folder on disk, and the oracle for them."""
import json
import os

import numpy as np

from oracle.latent_oracle import PepilixOracle
from seq2seqsharp_b200.pepilix import config_from_json, file_names
from seq2seqsharp_b200.safetensors_file import to_bfloat16, to_float32, write_safetensors


def layer(heads, dim, rot, vdim, rank, scale=0.3, base=10000.0, kv_from=None, experts=None, top=1, ff=24, limit=1.0):
    m = {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "kv_rank": rank, "scale": scale, "rot": {"base": base, "dims": rot}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    mlp = None
    if experts:
        mlp = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(layers, width, vocab, groups=1, taps=2, eps=1e-5, embed=1.0, logit=1.0):
    return {"architecture": "Pepilix", "canon": {"taps": taps}, "embedding": {"scale": embed}, "layers": layers, "logit_scale": logit,
            "norm": {"eps": eps, "groups": groups}, "vocab": vocab, "width": width}


CONFIGS = {
    # layers of unequal sizes, one without a feed-forward, caches read by later layers, two experts per token
    "mixed": config([layer(3, 16, 8, 24, 40, experts=5, top=2, ff=40), layer(2, 24, 8, 16, 40, kv_from=0, scale=0.5), layer(5, 8, 16, 8, 32, base=500.0, experts=3, ff=56, limit=0.6),
                     layer(4, 16, 16, 16, 32, base=500.0, kv_from=2, experts=7, top=3, ff=16)], 96, 101, groups=3, taps=3, embed=2.5, logit=0.7),
    # nothing is a multiple of eight: no tensor-core path takes these shapes
    "odd": config([layer(3, 10, 6, 9, 20, experts=4, top=2, ff=13), layer(1, 7, 2, 5, 20, experts=2, ff=9)], 50, 61, groups=5, taps=5, embed=3.0, logit=1.3),
    # one group, one tap, one head, every token uses every expert
    "plain": config([layer(1, 32, 32, 32, 64, experts=2, top=2, ff=32, limit=9.0)], 64, 73, groups=1, taps=1),
    # wide enough for every tensor-core kernel: expanded and absorbed attention, grouped products
    "wide": config([layer(8, 64, 32, 64, 128, scale=0.1, experts=6, top=2, ff=96), layer(8, 64, 32, 64, 128, scale=0.1, kv_from=0, experts=6, ff=96),
                    layer(2, 128, 64, 128, 320, scale=0.08)], 256, 300, groups=8, taps=4, embed=4.0, logit=2.0),
}


def weights(cfg, seed=1, std=0.25):
    """Tensor name -> float32 values that bfloat16 holds exactly (tables int32)."""
    rng = np.random.default_rng(seed)
    c = config_from_json(cfg)
    names = file_names(c)
    out = {}
    for engine, shape in c.weight_shapes().items():
        n = names[engine]
        if n.endswith("table"):
            x = c.layers[int(engine.split(".")[1])].experts
            out[n] = np.stack([rng.permutation(x.experts)[:x.top] for _ in range(shape[0])]).astype(np.int32)
            continue
        if "norm" in n:
            w = rng.uniform(0.5, 1.5, size=shape)
        elif n.endswith(".b"):
            w = rng.normal(0, 1.0, size=shape)
        elif "canon" in n:
            w = rng.normal(0, 0.5, size=shape)
        elif n == "embed":
            w = rng.normal(0, 1.0, size=shape)
        else:
            w = rng.normal(0, 1.0 / np.sqrt(shape[1]) * (std / 0.25), size=shape)
        a = to_float32(to_bfloat16(w.astype(np.float32)))
        out[n] = a.reshape(-1) if (shape[0] == 1 and ("norm" in n or n.endswith(".b"))) else a
    return out


def save(path, cfg, w):
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as fh:
        json.dump(cfg, fh)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v if v.dtype == np.int32 else to_bfloat16(v) for k, v in w.items()})
    return str(path)


def tokens(cfg, n, seed=0):
    return [int(t) for t in np.random.default_rng(1000 + seed).integers(1, cfg["vocab"], size=n)]


def oracle(cfg, w):
    return PepilixOracle(cfg, w)


def rel(got, want):
    """Largest root-mean-square difference of a row relative to the spread of all wanted values."""
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.sqrt(((got - want) ** 2).mean(axis=-1)).max() / want.std())


TOL = {"float32": 5e-6, "bfloat16": 4e-2}
