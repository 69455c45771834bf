"""Model classes by the ``architecture`` of a config file, and loading of a model folder (config.json and
model.safetensors).  A registered class has ``from_config(dict, device, dtype)`` and ``load_tensors(tensors)``."""
import importlib
import json
import os

import torch

from .weights import SafeTensors

# architecture -> "module:class"; imported on first use
_MODELS = {
    "Based": "based_b200.model:BasedLMHeadModel",
    "Razesun": "based_b200.razesun:RazesunLMHeadModel",
    "Vubenex": "based_b200.vubenex:VubenexLMHeadModel",
}
# architectures whose kernels are all in one part of the library (see build.PARTS)
_PARTS = {"Razesun": "hybrid", "Vubenex": "postnorm"}


def library_part(folder: str):
    """The part of the kernel library that the model in ``folder`` needs, None for the whole."""
    with open(os.path.join(folder, "config.json")) as f:
        return _PARTS.get(json.load(f).get("architecture"))


def architectures():
    return sorted(_MODELS)


def model_class(architecture: str):
    if architecture not in _MODELS:
        raise ValueError(f"unknown architecture {architecture!r} (known: {', '.join(architectures())})")
    module, name = _MODELS[architecture].split(":")
    return getattr(importlib.import_module(module), name)


def build_model(config: dict, device="cuda", dtype=torch.bfloat16):
    """The model a config describes, with uninitialised weights."""
    return model_class(config["architecture"]).from_config(config, device=device, dtype=dtype)


def load_model(folder: str, device="cuda", dtype=torch.bfloat16):
    """The model of a folder with config.json and model.safetensors, in eval mode, weights cast to ``dtype``."""
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    model = build_model(config, device=device, dtype=dtype)
    model.load_tensors(SafeTensors(os.path.join(folder, "model.safetensors")))
    return model.eval()
