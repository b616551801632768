"""Models whose layers are described one by one: configuration and host class.

`GPTConfig` (gpt.py) repeats one layer of one shape; a `LayeredConfig` lists its layers, each with a mixer and (or without) a
feed-forward.  The engine behind it is the same one (`TSB200_GptCreateLayered`), so a `LayeredGPT` is a `GPT`: prefill, decode, slots,
snapshots, KV pool, beam search, sampling and the slot scheduler work on it unchanged.
"""
import ctypes as C
from dataclasses import dataclass, field
from typing import Dict, List, Optional, Union

import numpy as np

from . import _native as N
from .gpt import GPT
from .synthetic import synth


def only_keys(d: dict, known, where: str):
    """For readers of model configurations: a key that is not known would change the model, so it is refused."""
    unknown = set(d) - set(known)
    if unknown:
        raise ValueError("%s: unknown keys %s" % (where, sorted(unknown)))


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
class GroupedAttention:
    """Attention with kv_heads key/value heads (query head h reads key/value head h // (heads // kv_heads)) over cached keys and values.
    score = scale q . k + bias[bucket(i - j)]; position i sees j <= i with i - j < window or j < keep_first."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float             # of the scores (not of the bias)
    window: int = 0          # 0: every earlier position
    keep_first: int = 0
    bias_rows: int = 0       # rows of the distance bias table, 0: none; half of them for single distances, half logarithmic up to bias_max
    bias_max: int = 0
    qk_norm: bool = False    # per-head RMS norm of queries and keys
    qkv_bias: bool = False
    sink: bool = False       # a logit per head that joins the softmax's denominator
    head_gate: bool = False  # head outputs times sigmoid(gate h)
    kv_from: int = -1        # attend to another layer's cache instead of an own one


@dataclass
class MatrixMemory:
    """Matrix memory with exponential gates (mLSTM): per head a state [dim, vdim] of fixed size instead of a cache."""
    heads: int
    dim: int
    vdim: int
    gate_cap: float          # soft cap of the gates' logits


@dataclass
class DenseGated:
    """down(silu(gate h) * up h)."""
    ff: int


@dataclass
class BlockLayer:
    mixer: Union[LatentAttention, GroupedAttention, MatrixMemory]
    experts: Optional[TableExperts] = None     # feed-forward of gated blocks
    dense: Optional[DenseGated] = None         # feed-forward of sandwich blocks


@dataclass
class LayeredConfig:
    d: int
    V: int
    layers: List[BlockLayer] = field(default_factory=list)
    block: str = "gated"        # "gated": latent attention and experts, parallel and gated; "sandwich": norms around every sublayer
    norm_groups: int = 1
    conv_taps: int = 1
    eps: float = 1e-6
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    tied_head: bool = True      # logits from the embedding table; False: a "head" matrix
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
        s = {"embed": (self.V, self.d), "final_norm": (1, self.d)}
        if not self.tied_head:
            s["head"] = (self.V, self.d)
        for i, layer in enumerate(self.layers):
            p = "layer.%d." % i
            s.update({p + n: v for n, v in (self._sandwich_shapes(layer) if self.block == "sandwich" else self._gated_shapes(layer)).items()})
        return s

    def _gated_shapes(self, layer) -> Dict[str, tuple]:
        d, m, x = self.d, layer.mixer, layer.experts
        s = {"norm1": (1, d), "conv1": (d, self.conv_taps), "gate1.w": (d, d), "gate1.b": (1, d), "attn.q": (m.heads * (m.dim + m.rot_dim), d)}
        if m.kv_from < 0:
            s["attn.dkv"], s["attn.dkv_norm"] = (m.kv_rank + m.rot_dim, d), (1, m.kv_rank)
        s["attn.uk"], s["attn.uv"] = (m.heads * m.dim, m.kv_rank), (m.heads * m.vdim, m.kv_rank)
        s["attn.o"] = (d, m.heads * m.vdim)
        if x is not None:
            s["norm2"], s["gate2.w"], s["gate2.b"] = (1, d), (d, d), (1, d)
            s["experts.table"] = (self.V, x.top)
            for e in range(x.experts):
                q = "experts.%d." % e
                s[q + "gate"], s[q + "up"], s[q + "down"] = (x.ff, d), (x.ff, d), (d, x.ff)
        return s

    def _sandwich_shapes(self, layer) -> Dict[str, tuple]:
        d, m = self.d, layer.mixer
        s = {"norm1": (1, d), "norm1b": (1, d), "scale1": (1, d)}
        if isinstance(m, GroupedAttention):
            own = m.kv_from < 0
            rows = {"q": m.heads * m.dim, **({"k": m.kv_heads * m.dim, "v": m.kv_heads * m.vdim} if own else {})}
            for n, r in rows.items():
                s["attn." + n] = (r, d)
                if m.qkv_bias:
                    s["attn.%s.b" % n] = (1, r)
                if m.qk_norm and n != "v":
                    s["attn.%s_norm" % n] = (1, m.dim)
            if m.bias_rows:
                s["attn.bias"] = (m.bias_rows, m.heads)
            if m.sink:
                s["attn.sink"] = (1, m.heads)
            if m.head_gate:
                s["attn.gate"] = (m.heads, d)
            s["attn.o"] = (d, m.heads * m.vdim)
        else:
            for n, r in (("q", m.heads * m.dim), ("k", m.heads * m.dim), ("v", m.heads * m.vdim), ("gate", m.heads * m.vdim), ("i", m.heads), ("f", m.heads)):
                s["mem." + n] = (r, d)
            s["mem.i.b"], s["mem.f.b"], s["mem.norm"] = (1, m.heads), (1, m.heads), (1, m.heads * m.vdim)
            s["mem.o"] = (d, m.heads * m.vdim)
        if layer.dense is not None:
            ff = layer.dense.ff
            s["norm2"], s["norm2b"], s["scale2"] = (1, d), (1, d), (1, d)
            s["ff.gate"], s["ff.up"], s["ff.down"] = (ff, d), (ff, d), (d, ff)
        return s

    def active_matmul_params(self) -> int:
        """Multiply-adds of the matrices per token (experts: the ones a token uses; keys and values once per position)."""
        n = 0
        for name, (r, c) in self.weight_shapes().items():
            layer = self.layers[int(name.split(".")[1])] if name.startswith("layer.") else None
            if name == "embed":
                n += r * c if self.tied_head else 0
            elif ".experts." in name:
                n += 0 if name.endswith("table") else r * c * layer.experts.top // layer.experts.experts
            elif r > 1 and not name.endswith(("conv1", "attn.bias")):
                n += r * c
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
        c.block, c.tied_head = {"gated": N.BLOCK_GATED, "sandwich": N.BLOCK_SANDWICH}[cfg.block], int(cfg.tied_head)
        descs = (N.LayerDescC * cfg.L)()
        for t, layer in zip(descs, cfg.layers):
            m, x = layer.mixer, layer.experts
            t.heads, t.dim, t.vdim, t.kv_from = m.heads, m.dim, m.vdim, -1
            if isinstance(m, LatentAttention):
                t.mixer, t.rot_dim, t.kv_rank = N.MIXER_LATENT, m.rot_dim, m.kv_rank
                t.rot_dims, t.kv_from, t.scale, t.rot_base = m.rot_dims, m.kv_from, m.scale, m.rot_base
            elif isinstance(m, GroupedAttention):
                t.mixer, t.kv_heads, t.scale, t.kv_from = N.MIXER_GROUPED, m.kv_heads, m.scale, m.kv_from
                t.window, t.keep_first, t.bias_rows, t.bias_max = m.window, m.keep_first, m.bias_rows, m.bias_max
                t.flags = (N.ATTN_QK_NORM * m.qk_norm) | (N.ATTN_QKV_BIAS * m.qkv_bias) | (N.ATTN_SINK * m.sink) | (N.ATTN_HEAD_GATE * m.head_gate)
            else:
                t.mixer, t.gate_cap = N.MIXER_MEMORY, m.gate_cap
            if x is not None:
                t.experts, t.top, t.ff = x.experts, x.top, x.ff
                t.glu_limit, t.glu_slope, t.glu_shift = x.limit, x.slope, x.shift
            elif layer.dense is not None:
                t.ff = layer.dense.ff
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
    """Seeded weights by engine name (float32 values that bfloat16 holds exactly): matrices N(0, std), norm gains and scales 1, biases N(0, bias_std)."""
    from .safetensors_file import to_bfloat16, to_float32
    rng = np.random.default_rng(seed)
    out = {}
    for name, shape in cfg.weight_shapes().items():
        if name.endswith("experts.table"):
            x = cfg.layers[int(name.split(".")[1])].experts
            out[name] = np.stack([rng.permutation(x.experts)[:x.top] for _ in range(shape[0])]).astype(np.int32)
            continue
        if "norm" in name or ".scale" in name:
            w = np.ones(shape, dtype=np.float32)
        elif name.endswith(".b"):
            w = synth(name, shape, seed, bias_std) if bias_std > 0 else np.zeros(shape, dtype=np.float32)
        else:
            w = synth(name, shape, seed, std)
        out[name] = to_float32(to_bfloat16(w))
    return out
