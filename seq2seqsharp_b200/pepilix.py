"""The decoder design "Pepilix" on the layered engine: config.json -> `LayeredConfig`, tensor names of model.safetensors -> engine names.

Per layer: latent attention behind a short causal convolution of its input and experts chosen by token id, both on group-wise
RMS norms of the same residual stream, each multiplied by a sigmoid gate of its own input before it is added.
"""
import re
from typing import Dict

from .layered import BlockLayer, LatentAttention, LayeredConfig, TableExperts, only_keys

ARCHITECTURE = "Pepilix"
# constants of the design's experts: hidden = a sigmoid(1.702 a) (u + 1)
EXPERT_SLOPE, EXPERT_SHIFT = 1.702, 1.0


def config_from_json(j: dict, dtype: str = "bfloat16") -> LayeredConfig:
    """The parsed config.json as a `LayeredConfig`.  Unknown kinds and keys are refused: they would change the model."""
    if j.get("architecture") != ARCHITECTURE:
        raise ValueError("not a %s model: architecture %r" % (ARCHITECTURE, j.get("architecture")))
    only_keys(j, ("architecture", "canon", "embedding", "layers", "logit_scale", "norm", "vocab", "width"), "config.json")
    cfg = LayeredConfig(d=int(j["width"]), V=int(j["vocab"]), norm_groups=int(j["norm"]["groups"]), conv_taps=int(j["canon"]["taps"]),
                        eps=float(j["norm"]["eps"]), embed_scale=float(j["embedding"]["scale"]), logit_scale=float(j["logit_scale"]), dtype=dtype,
                        name=ARCHITECTURE)
    for i, layer in enumerate(j["layers"]):
        where = "layer %d" % i
        only_keys(layer, ("type", "mixer", "mlp"), where)
        if layer["type"] != "latent_attention":
            raise ValueError("%s: unknown type %r" % (where, layer["type"]))
        m = layer["mixer"]
        only_keys(m, ("dim", "heads", "kv_rank", "rot", "rot_dim", "scale", "vdim", "kv_from"), where + " mixer")
        only_keys(m["rot"], ("base", "dims"), where + " rotation")
        src = m.get("kv_from")
        mixer = LatentAttention(heads=int(m["heads"]), dim=int(m["dim"]), rot_dim=int(m["rot_dim"]), vdim=int(m["vdim"]), kv_rank=int(m["kv_rank"]),
                                rot_base=float(m["rot"]["base"]), rot_dims=int(m["rot"]["dims"]), scale=float(m["scale"]),
                                kv_from=-1 if src is None else int(src))
        experts = None
        if layer.get("mlp") is not None:
            f = layer["mlp"]
            only_keys(f, ("kind", "expert", "router"), where + " mlp")
            if f.get("kind", "moe") != "moe":
                raise ValueError("%s: unknown feed-forward %r" % (where, f["kind"]))
            only_keys(f["expert"], ("ff", "limit"), where + " expert")
            only_keys(f["router"], ("experts", "top"), where + " router")
            experts = TableExperts(experts=int(f["router"]["experts"]), top=int(f["router"]["top"]), ff=int(f["expert"]["ff"]),
                                   limit=float(f["expert"]["limit"]), slope=EXPERT_SLOPE, shift=EXPERT_SHIFT)
        cfg.layers.append(BlockLayer(mixer, experts))
    return cfg


_PLAIN = {"norm1": "norm1", "norm2": "norm2", "canon1": "conv1", "rg1": "gate1.w", "rg1.b": "gate1.b", "rg2": "gate2.w", "rg2.b": "gate2.b",
          "mix.q": "attn.q", "mix.dkv": "attn.dkv", "mix.dkv.norm": "attn.dkv_norm", "mix.uk": "attn.uk", "mix.uv": "attn.uv", "mix.o": "attn.o",
          "mlp.table": "experts.table"}


def engine_name(name: str) -> str:
    """Engine weight name of a tensor of the file; KeyError for names the design does not have."""
    if name == "embed":
        return "embed"
    if name == "final.norm":
        return "final_norm"
    m = re.fullmatch(r"l(\d+)\.(.+)", name)
    if m is None:
        raise KeyError(name)
    e = re.fullmatch(r"mlp\.e(\d+)\.(gate|up|down)", m.group(2))
    if e is not None:
        return "layer.%s.experts.%s.%s" % (m.group(1), e.group(1), e.group(2))
    return "layer.%s.%s" % (m.group(1), _PLAIN[m.group(2)])


def file_names(cfg: LayeredConfig) -> Dict[str, str]:
    """Engine weight name -> tensor name in the file."""
    back = {v: k for k, v in _PLAIN.items()}
    out = {}
    for n in cfg.weight_shapes():
        if n in ("embed", "final_norm"):
            out[n] = {"embed": "embed", "final_norm": "final.norm"}[n]
            continue
        _, i, rest = n.split(".", 2)
        e = re.fullmatch(r"experts\.(\d+)\.(gate|up|down)", rest)
        out[n] = "l%s.%s" % (i, "mlp.e%s.%s" % e.groups() if e else back[rest])
    return out
