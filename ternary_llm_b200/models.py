"""Registry of the model designs the decoder serves, and loading by what is on disk.

A model on disk is either a `.tllm` file (the reference's container: the LLaMA design on
ternary weights) or a folder with config.json and model.safetensors, whose "architecture"
names the design.  load() returns a model object; Decoder (decoder.py) takes it, or the path.

A design adds itself with @register(name): a class with
    from_config(cfg: dict, tensors) -> model      (tensors: a mapping name -> array)
and, on the instance, what Decoder asks for: vocab_size, and create(decoder_args) (see
mixed.MixedModel for designs made of mixer layers).
"""
from __future__ import annotations

import json
import os

ARCHITECTURES: dict = {}


def register(name: str):
    def deco(cls):
        ARCHITECTURES[name] = cls
        cls.architecture = name
        return cls
    return deco


def load(path: str):
    """The model at `path`: a .tllm file or a folder with config.json and model.safetensors."""
    from . import mixed  # noqa: F401  (registers its designs)
    if not os.path.isdir(path):
        from .tllm_format import read_tllm
        return read_tllm(path)
    with open(os.path.join(path, "config.json")) as f:
        cfg = json.load(f)
    arch = cfg.get("architecture")
    if arch not in ARCHITECTURES:
        raise ValueError(f"{path}: unknown architecture {arch!r} (known: {', '.join(sorted(ARCHITECTURES))}, and .tllm files)")
    from .safetensors_io import SafetensorsFile
    return ARCHITECTURES[arch].from_config(cfg, SafetensorsFile(os.path.join(path, "model.safetensors")))
