"""Model registry: a configuration's `architecture` names the class that reads it.

A model class provides
    from_config(config, weights, device, dtype)   weights: checkpoint.Weights, or None for random ones
and its instances what the engine drives:
    device, vocab, num_layers, page_size (preferred), tau, seed
    make_caches(num_pages, page_size, max_len)     the step's cache, whatever the model keeps per token
    make_prefix(max_len) / None                    scratch for the prefilling entries' cached tokens, if it wants one
    step(caches, inp, ids, cached_lens, block_table, num_decoding, prefix) -> StepOutput
    logits(hidden)                                 fp32 or bf16 logits of normed rows
A class with `stateful = True` keeps a state per request beside the pages: its make_caches takes slots=, the number of state
slots, and its step slots=, int32 [entries], the slot of every entry (-1: padding).
"""
from __future__ import annotations

from dataclasses import dataclass

import torch

MODELS: dict[str, type] = {}


@dataclass
class StepOutput:
    tokens: torch.Tensor  # int64 [entries]: the sampled next token of every entry
    hidden: torch.Tensor  # [rows, width]: the final normed state of every packed row of the step


def register(architecture: str):
    def add(cls):
        MODELS[architecture] = cls
        return cls

    return add


def load_all() -> dict[str, type]:
    """Import every model module (each registers itself)."""
    from .. import scaffold  # noqa: F401  (registers itself)
    from . import biranex, radivik  # noqa: F401

    return MODELS


def model_class(config: dict) -> type:
    load_all()
    name = config.get("architecture")
    if name not in MODELS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(MODELS))}")
    return MODELS[name]


def load_model(folder: str, device="cuda", dtype: torch.dtype = torch.bfloat16, random_weights: bool = False):
    """The model of a folder (config.json + safetensors).  random_weights: from the configuration alone."""
    from .. import checkpoint

    config = checkpoint.read_config(folder)
    weights = None if random_weights else checkpoint.Weights.open(folder)
    return model_class(config).from_config(config, weights, torch.device(device), dtype)
