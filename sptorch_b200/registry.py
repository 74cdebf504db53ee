"""Which class runs which architecture, and loading a model folder (config.json + model.safetensors) through it."""
from __future__ import annotations

import json
import os

from . import weights
from .backend import BF16, FfiBackend
from .gpt import GPT, QwenLikeGPT
from .layered import DESIGNS, ConfigError, LayeredGPT


def _gpt_like(cls, eps):
    def build(backend, config, shapes, seq_len, dtype, max_batch):
        extra = {"rope_base": float(config["rope_base"])} if cls is QwenLikeGPT and "rope_base" in config else {}
        longest = int(config["seq_len"])
        return cls(backend, int(config["vocab"]), int(config["d_model"]), int(config["n_head"]), int(config["n_layer"]), int(config["d_ff"]),
                   longest if cls is GPT or not seq_len else min(seq_len, longest), dtype=dtype, max_batch=max_batch, eps=float(config.get("eps", eps)), **extra)
    return build


def _layered(backend, config, shapes, seq_len, dtype, max_batch):
    return LayeredGPT(backend, config, seq_len or int(config.get("seq_len", 4096)), dtype=dtype, max_batch=max_batch, shapes=shapes)


ARCHITECTURES = {"GPT": _gpt_like(GPT, 1e-5), "QwenLikeGPT": _gpt_like(QwenLikeGPT, 1e-6), **{name: _layered for name in DESIGNS}}


def read_config(folder: str) -> dict:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        config = json.load(f)
    arch = config.get("architecture")
    if arch not in ARCHITECTURES:
        raise ConfigError(f"config.json: architecture {arch!r} is not one of {sorted(ARCHITECTURES)}")
    return config


def load_model(backend: FfiBackend, folder: str, seq_len: int = 0, dtype: int = BF16, max_batch: int = 1):
    """The model of ``folder`` on the device: the class its config.json names, its tensors from model.safetensors.  ``seq_len``: the
    most positions a sequence may have (0: the configuration's own)."""
    config = read_config(folder)
    with weights.WeightFile(os.path.join(folder, "model.safetensors"), weights.SAFETENSORS) as w:
        model = ARCHITECTURES[config["architecture"]](backend, config, w.shapes(), seq_len, dtype, max_batch)
        try:
            weights.load_into(model, w)
        except Exception:
            model.close()
            raise
    return model
