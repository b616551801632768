"""The decoder design "Gunuvik" on the layered engine: config.json and tensor shapes -> `LayeredConfig`, tensor names of
model.safetensors -> engine names.

Sandwich blocks: every sublayer stands between two norms and its result is scaled element by element.  Mixers: windowed grouped-query
attention without rotation (distance bias, sink, gated heads, caches shared between layers) and matrix memories; dense gated feed-forwards.
"""
import re
from typing import Dict, Mapping, Optional

from .layered import BlockLayer, DenseGated, GroupedAttention, LayeredConfig, MatrixMemory, only_keys

ARCHITECTURE = "Gunuvik"


def _attention(m: dict, where: str, rel_rows: int) -> GroupedAttention:
    only_keys(m, ("bias_max", "dim", "heads", "kv_heads", "mask", "scale", "vdim", "kv_from"), where + " mixer")
    only_keys(m["mask"], ("size", "keep_first"), where + " mask")
    src = m.get("kv_from")
    if int(m["mask"]["size"]) < 1:
        raise ValueError("%s: a window of %r positions" % (where, m["mask"]["size"]))
    return GroupedAttention(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), scale=float(m["scale"]),
                            window=int(m["mask"]["size"]), keep_first=int(m["mask"]["keep_first"]), bias_rows=rel_rows, bias_max=int(m["bias_max"]),
                            qk_norm=True, qkv_bias=True, sink=True, head_gate=True, kv_from=-1 if src is None else int(src))


def config_from_json(j: dict, dtype: str = "bfloat16", shapes: Optional[Mapping[str, tuple]] = None) -> LayeredConfig:
    """The parsed config.json as a `LayeredConfig`; `shapes` are the tensors' (the distance bias tables say their size only there).
    Unknown kinds and keys are refused: they would change the model."""
    if j.get("architecture") != ARCHITECTURE:
        raise ValueError("not a %s model: architecture %r" % (ARCHITECTURE, j.get("architecture")))
    only_keys(j, ("architecture", "embedding", "layers", "norm", "vocab", "width"), "config.json")
    only_keys(j["embedding"], ("scale",), "embedding")
    only_keys(j["norm"], ("eps",), "norm")
    cfg = LayeredConfig(d=int(j["width"]), V=int(j["vocab"]), block="sandwich", eps=float(j["norm"]["eps"]), embed_scale=float(j["embedding"]["scale"]),
                        tied_head=False, dtype=dtype, name=ARCHITECTURE)
    for i, layer in enumerate(j["layers"]):
        where = "layer %d" % i
        only_keys(layer, ("type", "mixer", "mlp"), where)
        m = layer["mixer"]
        if layer["type"] == "attention":
            rel = "l%d.mix.rel" % i
            if shapes is None or rel not in shapes:
                raise ValueError("%s: the shape of %s is needed" % (where, rel))
            mixer = _attention(m, where, int(shapes[rel][0]))
        elif layer["type"] == "mlstm":
            only_keys(m, ("dim", "gate_cap", "heads", "vdim"), where + " mixer")
            mixer = MatrixMemory(heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), gate_cap=float(m["gate_cap"]))
        else:
            raise ValueError("%s: unknown type %r" % (where, layer["type"]))
        dense = None
        if layer.get("mlp") is not None:
            only_keys(layer["mlp"], ("kind", "ff"), where + " mlp")
            if layer["mlp"].get("kind", "dense") != "dense":
                raise ValueError("%s: unknown feed-forward %r" % (where, layer["mlp"]["kind"]))
            dense = DenseGated(int(layer["mlp"]["ff"]))
        cfg.layers.append(BlockLayer(mixer, dense=dense))
    return cfg


_ATTENTION = {"mix.q": "attn.q", "mix.k": "attn.k", "mix.v": "attn.v", "mix.q.b": "attn.q.b", "mix.k.b": "attn.k.b", "mix.v.b": "attn.v.b",
              "mix.q.norm": "attn.q_norm", "mix.k.norm": "attn.k_norm", "mix.rel": "attn.bias", "mix.sink": "attn.sink", "mix.g": "attn.gate", "mix.o": "attn.o"}
_MEMORY = {"mix.q": "mem.q", "mix.k": "mem.k", "mix.v": "mem.v", "mix.g": "mem.gate", "mix.i": "mem.i", "mix.f": "mem.f", "mix.i.b": "mem.i.b",
           "mix.f.b": "mem.f.b", "mix.norm": "mem.norm", "mix.o": "mem.o"}
_PLAIN = {"norm1": "norm1", "norm1b": "norm1b", "ls1": "scale1", "norm2": "norm2", "norm2b": "norm2b", "ls2": "scale2", "mlp.gate": "ff.gate",
          "mlp.up": "ff.up", "mlp.down": "ff.down"}
_TOP = {"embed": "embed", "final.norm": "final_norm", "head": "head"}


def engine_name(name: str, cfg: LayeredConfig) -> str:
    """Engine weight name of a tensor of the file; KeyError for names the design does not have."""
    if name in _TOP:
        return _TOP[name]
    m = re.fullmatch(r"l(\d+)\.(.+)", name)
    if m is None or int(m.group(1)) >= cfg.L:
        raise KeyError(name)
    mix = _ATTENTION if isinstance(cfg.layers[int(m.group(1))].mixer, GroupedAttention) else _MEMORY
    return "layer.%s.%s" % (m.group(1), {**_PLAIN, **mix}[m.group(2)])


def file_names(cfg: LayeredConfig) -> Dict[str, str]:
    """Engine weight name -> tensor name in the file."""
    back = {v: k for d in (_ATTENTION, _MEMORY, _PLAIN) for k, v in d.items()}
    top = {v: k for k, v in _TOP.items()}
    out = {}
    for n in cfg.weight_shapes():
        out[n] = top[n] if n in top else "l%s.%s" % (n.split(".")[1], back[n.split(".", 2)[2]])
    return out
