"""Models by the name their config.json gives (`architecture`), and loading one from a folder with config.json and
model.safetensors.

A registered class has ``from_config(dict) -> config``, ``__init__(config, weights, device, dtype)`` with `weights` a
``checkpoint.Checkpoint`` (or any mapping), ``new_cache(max_batch, max_seq_len, num_pages)`` for the KV manager that
fits it, and the ``inference`` / ``next_tokens`` methods that ``Engine`` drives."""
from __future__ import annotations

import json
from pathlib import Path

import torch

from .checkpoint import Checkpoint
from .gifetar import Gifetar
from .munadra import Munadra

MODELS = {"Gifetar": Gifetar, "Munadra": Munadra}


def model_class(config: dict):
    """The class registered for a config.json's architecture."""
    name = config.get("architecture")
    if name not in MODELS:
        raise KeyError(f"unknown architecture {name!r}; known: {sorted(MODELS)}")
    return MODELS[name]


def load_config(path):
    """(model class, its config object) of a model folder."""
    with open(Path(path) / "config.json") as f:
        raw = json.load(f)
    cls = model_class(raw)
    return cls, cls.from_config(raw)


def load_model(path, device="cuda:0", dtype=torch.bfloat16):
    """Model folder -> model with its weights on `device`."""
    cls, config = load_config(path)
    weights = Checkpoint(Path(path) / "model.safetensors")
    model = cls(config, weights, device, dtype)
    if weights.unread():
        raise ValueError(f"{path}: tensors that the architecture does not know: {weights.unread()[:5]}")
    return model
