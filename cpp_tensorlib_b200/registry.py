"""Model registry: the architecture a folder's config.json names -> the class that runs it.

An entry is "module:class"; the class has ``from_folder(config, tensors, dtype, max_ctx)`` and is a
``Sequence``.  Modules are imported on use (the int4 decoder needs torch, the layer stack does not).
"""
import importlib
import json
import os

from .safetensors import SafeTensors

ARCHITECTURES = {
    "Qwen2ForCausalLM": "cpp_tensorlib_b200.decoder:Q4Decoder",
    "Zavilorn": "cpp_tensorlib_b200.zavilorn:Zavilorn",
    "Daronex": "cpp_tensorlib_b200.daronex:Daronex",
}
DTYPES = ("bfloat16", "float32")


def architecture(config):
    name = config.get("architecture") or (config.get("architectures") or [None])[0]
    if name not in ARCHITECTURES:
        raise ValueError(f"config.json names no known architecture ({name!r}; known: {sorted(ARCHITECTURES)})")
    return name


def model_class(config):
    module, cls = ARCHITECTURES[architecture(config)].split(":")
    return getattr(importlib.import_module(module), cls)


def load_model(folder, dtype="bfloat16", max_ctx=4096):
    """The model of `folder` (config.json, model.safetensors), ready for a sequence of `max_ctx` tokens."""
    if dtype not in DTYPES:
        raise ValueError(f"dtype must be one of {DTYPES}")
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    tensors = SafeTensors(os.path.join(folder, "model.safetensors"))
    return model_class(config).from_folder(config, tensors, dtype, max_ctx)
