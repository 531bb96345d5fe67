"""The model families and how a checkpoint folder names one.

``load(ctx, folder, ...)`` reads ``config.json``, picks the family and returns the model on the device; every model takes
ragged steps (``step``), has pools of its geometry (``kv_pool``, ``state_pool``) and runs in :class:`engine.Engine`.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass
from typing import Callable

from . import api
from .loader import QUANT_F32, LayeredConfig, LlamaConfig, load_weights, read_safetensors


@dataclass
class Family:
    """``load(ctx, folder, config dict, dtype, max_rows, quantization)`` -> model; ``dtypes`` it computes in (first: default)."""

    load: Callable
    dtypes: tuple


def _weights_file(folder: str) -> str:
    return os.path.join(folder, "model.safetensors")


def _load_llama(ctx, folder, config, dtype, max_rows, quantization):
    cfg = LlamaConfig.from_hf_config(os.path.join(folder, "config.json"))
    cfg.quantization = quantization
    return api.LlamaWeights(ctx, cfg, load_weights(_weights_file(folder), cfg), max_batch=max_rows)


def _layered(read_config):
    def load(ctx, folder, config, dtype, max_rows, quantization):
        if quantization != QUANT_F32:
            raise ValueError("this design keeps its bf16 weights: quantization is not offered")
        return api.LayeredModel(ctx, read_config(config), read_safetensors(_weights_file(folder)), dtype, max_rows)
    return load


FAMILIES = {
    # activations and KV are f32 throughout, the bf16 checkpoint widens exactly
    "Llama": Family(_load_llama, ("float32",)),
    "Sumosun": Family(_layered(LayeredConfig.from_sumosun), ("bfloat16", "float32")),
    "Lilosun": Family(_layered(LayeredConfig.from_lilosun), ("bfloat16", "float32")),
    "Rubuvik": Family(_layered(LayeredConfig.from_rubuvik), ("bfloat16", "float32")),
    "Noresun": Family(_layered(LayeredConfig.from_noresun), ("bfloat16", "float32")),
}


def family_of(config: dict) -> str:
    """The family's name: the key "architecture", or HuggingFace's "architectures" / "model_type"; a config that names
    nothing is a Llama (the reference's loader knows no other)."""
    name = config.get("architecture") or (config.get("architectures") or [None])[0] or config.get("model_type") or "Llama"
    for family in FAMILIES:
        if name.lower().startswith(family.lower()):
            return family
    raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(FAMILIES))}")


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json")) as f:
        return json.load(f)


def load(ctx, folder: str, dtype: str | None = None, max_rows: int = 64, quantization: str = QUANT_F32):
    """The checkpoint in ``folder`` on the device.  ``max_rows``: tokens one batched step can take."""
    config = read_config(folder)
    family = FAMILIES[family_of(config)]
    dtype = dtype or family.dtypes[0]
    if dtype not in family.dtypes:
        raise UnsupportedDtype(f"{family_of(config)} computes in {' or '.join(family.dtypes)}, not in {dtype}")
    return family.load(ctx, folder, config, dtype, max_rows, quantization)


class UnsupportedDtype(ValueError):
    pass
