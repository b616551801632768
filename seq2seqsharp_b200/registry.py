"""Model registry: which class and which loader serve a model on disk.

A folder with config.json and model.safetensors is served by the design its "architecture" names (`ARCHITECTURES`); a file is the
reference's protobuf model file (model_file.py).  `load_model` is what the command line, the trace runner and servers call.
"""
import json
import os
from dataclasses import dataclass
from typing import Callable, Dict, Mapping

from . import gunuvik, pepilix
from .layered import LayeredConfig, LayeredGPT
from .safetensors_file import SafetensorsFile


@dataclass
class Architecture:
    config: Callable[[dict, str, Mapping], LayeredConfig]     # (config.json, dtype, tensor shapes of the file) -> configuration
    tensor_name: Callable[[str, LayeredConfig], str]          # tensor name in the file -> engine name
    dtypes: tuple = ("bfloat16", "float32")


ARCHITECTURES: Dict[str, Architecture] = {
    pepilix.ARCHITECTURE: Architecture(lambda j, dtype, shapes: pepilix.config_from_json(j, dtype), lambda n, cfg: pepilix.engine_name(n)),
    gunuvik.ARCHITECTURE: Architecture(gunuvik.config_from_json, gunuvik.engine_name),
}


def weights_file(path: str) -> SafetensorsFile:
    return SafetensorsFile(os.path.join(path, "model.safetensors"))


def read_config(path: str, dtype: str = "bfloat16"):
    """(architecture, configuration) of a model folder."""
    with open(os.path.join(path, "config.json"), encoding="utf-8") as fh:
        j = json.load(fh)
    name = j.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError("no such architecture: %r (known: %s)" % (name, ", ".join(sorted(ARCHITECTURES))))
    arch = ARCHITECTURES[name]
    if dtype not in arch.dtypes:
        raise ValueError("%s models are not served in %s" % (name, dtype))
    tensors = weights_file(path)
    return arch, arch.config(j, dtype, {n: tensors.shape(n) for n in tensors.names()})


def load_model(path: str, dtype: str = "bfloat16", device_id: int = 0, max_batch: int = 1, max_tokens: int = 512):
    """An engine with the model's weights, ready to run."""
    if os.path.isdir(path):
        arch, cfg = read_config(path, dtype)
        tensors = weights_file(path)
        names = {arch.tensor_name(n, cfg): n for n in tensors.names()}
        missing = sorted(set(cfg.weight_shapes()) - set(names))
        if missing:
            raise ValueError("%s: %d tensors are missing, the first is %s" % (tensors.path, len(missing), missing[0]))
        gpt = LayeredGPT(cfg, device_id=device_id, max_batch=max_batch, max_tokens=max_tokens)
        for engine in cfg.weight_shapes():
            gpt.SetWeight(engine, tensors.get(names[engine]))
        return gpt
    from .model_file import load_gpt
    return load_gpt(path, device_id=device_id, max_batch=max_batch, max_tokens=max_tokens, dtype="float32" if dtype == "float32" else None)[0]
