"""Models whose layers are described one by one: configuration and host class.

`GPTConfig` (gpt.py) repeats one layer of one shape; a `LayeredConfig` lists its layers, each with a mixer and (or without) a
feed-forward.  The engine behind it is the same one (`TSB200_GptCreateLayered`), so a `LayeredGPT` is a `GPT`: prefill, decode, slots,
snapshots, KV pool, beam search, sampling and the slot scheduler work on it unchanged.
"""
import ctypes as C
from dataclasses import dataclass, field
from typing import Dict, List, Optional

import numpy as np

from . import _native as N
from .gpt import GPT
from .synthetic import synth


@dataclass
class LatentAttention:
    """Attention over one cached vector per position: a normed latent and a rotated key part shared by all heads."""
    heads: int
    dim: int                 # unrotated query/key size of a head
    rot_dim: int             # rotated query/key size
    vdim: int
    kv_rank: int             # size of the latent
    rot_base: float
    scale: float             # of the scores
    rot_dims: int = 0        # how many of the rotated dimensions turn (0: all)
    kv_from: int = -1        # attend to another layer's cache instead of an own one

    def __post_init__(self):
        self.rot_dims = self.rot_dims or self.rot_dim


@dataclass
class TableExperts:
    """Gated feed-forward experts chosen by token id; each of the `top` experts of a token has weight 1 / top.
    a = min(gate, limit), u = clamp(up, -limit, limit), hidden = a sigmoid(slope a) (u + shift)."""
    experts: int
    top: int
    ff: int
    limit: float
    slope: float
    shift: float


@dataclass
class BlockLayer:
    mixer: LatentAttention
    experts: Optional[TableExperts] = None


@dataclass
class LayeredConfig:
    d: int
    V: int
    layers: List[BlockLayer] = field(default_factory=list)
    norm_groups: int = 1
    conv_taps: int = 1
    eps: float = 1e-6
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    dtype: str = "bfloat16"     # "bfloat16" | "float32"
    name: str = ""
    # what a GPTConfig would say here: no attention over an encoder, no position table (positions are the mixers' business)
    cross_attn = False
    pe = 0
    ape_decode_pos0 = False

    @property
    def L(self):
        return len(self.layers)

    def weight_shapes(self) -> Dict[str, tuple]:
        """Engine weight names -> shapes ([out, in] for matrices)."""
        d, V = self.d, self.V
        s = {"embed": (V, d), "final_norm": (1, d)}
        for i, layer in enumerate(self.layers):
            p, m, x = "layer.%d." % i, layer.mixer, layer.experts
            s[p + "norm1"], s[p + "conv1"], s[p + "gate1.w"], s[p + "gate1.b"] = (1, d), (d, self.conv_taps), (d, d), (1, d)
            s[p + "attn.q"] = (m.heads * (m.dim + m.rot_dim), d)
            if m.kv_from < 0:
                s[p + "attn.dkv"], s[p + "attn.dkv_norm"] = (m.kv_rank + m.rot_dim, d), (1, m.kv_rank)
            s[p + "attn.uk"], s[p + "attn.uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
            s[p + "attn.o"] = (d, m.heads * m.vdim)
            if x is not None:
                s[p + "norm2"], s[p + "gate2.w"], s[p + "gate2.b"] = (1, d), (d, d), (1, d)
                s[p + "experts.table"] = (V, x.top)
                for e in range(x.experts):
                    q = p + "experts.%d." % e
                    s[q + "gate"], s[q + "up"], s[q + "down"] = (x.ff, d), (x.ff, d), (d, x.ff)
        return s

    def active_matmul_params(self) -> int:
        """Multiply-adds of the matrices per token (experts: the ones a token uses; keys and values once per position)."""
        n = self.d * self.V
        for layer in self.layers:
            m, x = layer.mixer, layer.experts
            n += self.d * self.d * (2 if x is not None else 1) + self.d * m.heads * (m.dim + m.rot_dim) + m.heads * m.vdim * self.d
            n += m.heads * (m.dim + m.vdim) * m.kv_rank
            if m.kv_from < 0:
                n += self.d * (m.kv_rank + m.rot_dim)
            if x is not None:
                n += 3 * self.d * x.ff * x.top
        return n


class LayeredGPT(GPT):
    """One replica of a layered model on one device."""

    def __init__(self, cfg: LayeredConfig, device_id: int = 0, max_batch: int = 1, max_tokens: int = 512):
        self.cfg, self.device_id, self.max_batch, self.max_tokens = cfg, device_id, max_batch, max_tokens
        self._comm, self.tp_rank, self.tp_size = C.c_void_p(), 0, 1
        self._keep, self._B = None, 0
        c = N.LayeredConfigC()
        c.L, c.d, c.V = cfg.L, cfg.d, cfg.V
        c.dtype = {"bfloat16": N.BF16, "float32": N.F32}[cfg.dtype]
        c.norm_groups, c.conv_taps = cfg.norm_groups, cfg.conv_taps
        c.eps, c.embed_scale, c.logit_scale = cfg.eps, cfg.embed_scale, cfg.logit_scale
        c.max_batch, c.max_tokens, c.device = max_batch, max_tokens, device_id
        descs = (N.LayerDescC * cfg.L)()
        for t, layer in zip(descs, cfg.layers):
            m, x = layer.mixer, layer.experts
            t.mixer, t.heads, t.dim, t.rot_dim, t.vdim, t.kv_rank = 0, m.heads, m.dim, m.rot_dim, m.vdim, m.kv_rank
            t.rot_dims, t.kv_from, t.scale, t.rot_base = m.rot_dims, m.kv_from, m.scale, m.rot_base
            if x is not None:
                t.experts, t.top, t.ff = x.experts, x.top, x.ff
                t.glu_limit, t.glu_slope, t.glu_shift = x.limit, x.slope, x.shift
        self._h = C.c_void_p()
        N.call("TSB200_GptCreateLayered", C.byref(c), descs, C.byref(self._h))

    def LoadWeights(self, weights: Dict[str, np.ndarray]):
        """Tensors by engine name: float32, int32 (tables) or uint16 arrays (bfloat16 bit patterns)."""
        for name, w in weights.items():
            self.SetWeight(name, w)

    def SetWeight(self, name: str, w: np.ndarray):
        w = np.ascontiguousarray(w)
        dt = {np.dtype("uint16"): N.BF16, np.dtype("int32"): N.I32}.get(w.dtype)
        if dt is None:
            w, dt = w.astype(np.float32, copy=False), N.F32
        rows, cols = w.shape if w.ndim == 2 else (1, w.size)
        N.call("TSB200_GptSetWeight", self._h, name.encode(), w.ctypes.data_as(C.c_void_p), dt, rows, cols, 0)


def synthetic_layered_weights(cfg: LayeredConfig, seed: int, std: float = 0.02, bias_std: float = 0.0):
    """Seeded weights by engine name (float32 values that bfloat16 holds exactly): matrices N(0, std), norm gains 1, biases N(0, bias_std)."""
    from .safetensors_file import to_bfloat16, to_float32
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in cfg.weight_shapes().items():
        if name.endswith("experts.table"):
            x = cfg.layers[int(name.split(".")[1])].experts
            out[name] = np.stack([rng.permutation(x.experts)[:x.top] for _ in range(shape[0])]).astype(np.int32)
            continue
        if name == "final_norm" or name.endswith(("norm1", "norm2", "dkv_norm")):
            w = np.ones(shape, dtype=np.float32)
        elif name.endswith(".b"):
            w = synth(name, shape, seed, bias_std) if bias_std > 0 else np.zeros(shape, dtype=np.float32)
        else:
            w = synth(name, shape, seed, std)
        out[name] = to_float32(to_bfloat16(w))
    return out
