"""Which decoder class serves a model, by its configuration.

A model is a folder with ``config.json`` (whose "architecture" names the design) and ``model.safetensors``, or the reference's
weight file with its ``GptConfig`` JSON beside it (nn_b200.weights).
"""
from __future__ import annotations

import json
import os

from . import native as N
from .device import Device

DTYPES = {"bfloat16": N.NS_BF16, "float32": N.NS_F32}


def _fabezen():
    from .fabezen import Fabezen, FabezenConfig

    return Fabezen, FabezenConfig


def _topidra():
    from .topidra import Topidra, TopidraConfig

    return Topidra, TopidraConfig


# name -> () -> (decoder class, configuration class)
ARCHITECTURES = {"Fabezen": _fabezen, "Topidra": _topidra}


def _load_folder(dev: Device, folder: str, config: dict, dtype: str, batch: int, max_prefill: int, slots: int | None):
    from .weights import SafeTensors, check_shapes

    model_class, config_class = ARCHITECTURES[config["architecture"]]()
    cfg = config_class.from_dict(config)
    tensors = SafeTensors(os.path.join(folder, "model.safetensors"))
    check_shapes(tensors, cfg.tensor_shapes())
    return model_class(dev, cfg, tensors, batch=batch, max_prefill=max_prefill, dtype=DTYPES[dtype], slots=slots)


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        return json.load(f)


def load_model(dev: Device, path: str, dtype: str = "bfloat16", batch: int = 1, max_prefill: int = 512, slots: int | None = None):
    """A decoder for the model at `path`.  dtype "bfloat16": the serving precision of its class (for the reference's GPT files
    that is the int8 / bf16 decoder); "float32": everything in 32-bit."""
    if dtype not in DTYPES:
        raise ValueError(f"dtype {dtype!r}: one of {', '.join(DTYPES)}")
    if os.path.isdir(path):
        config = read_config(path)
        name = config.get("architecture")
        if name not in ARCHITECTURES:
            raise ValueError(f"{path}: architecture {name!r} is none of {', '.join(sorted(ARCHITECTURES))}")
        return _load_folder(dev, path, config, dtype, batch, max_prefill, slots)
    from .gpt import GptW8A8
    from .gpt_f32 import GptF32
    from .weights import load_char_gpt

    cfg, weights, _ = load_char_gpt(path)
    if dtype == "float32":
        return GptF32(dev, cfg, weights, batch, min(max_prefill, cfg.context))
    return GptW8A8(dev, cfg, weights, batch, min(max_prefill, cfg.context))
