"""Loading a checkpoint folder (``config.json`` + ``model.safetensors``) for inference.

``config.json`` names its architecture; the registry below maps the name to the module that builds the
model's configuration and its parameter tree.
"""

from __future__ import annotations

import importlib
import json
import os
from typing import Any, NamedTuple

import torch

from axlearn_b200.common import causal_lm
from axlearn_b200.common.safetensors_io import read_safetensors

# architecture -> module with ``checkpoint_model_config(config, tensors)`` and
# ``parameters(model, tensors, dtype=, device=)`` and ``KERNEL_SOURCES``.
ARCHITECTURES = {
    "Sagisun": "axlearn_b200.experiments.text.gpt.sagisun",
    "Zukitar": "axlearn_b200.experiments.text.gpt.zukitar",
}


class LoadedModel(NamedTuple):
    model: causal_lm.Model
    parameters: dict
    config: dict
    dtype: torch.dtype

    @property
    def decoder(self):
        return self.model.decoder


def load_model(folder: str, *, dtype: torch.dtype = torch.bfloat16, device: Any = None) -> LoadedModel:
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as f:
        config = json.load(f)
    name = config.get("architecture")
    if name not in ARCHITECTURES:
        raise ValueError(f"unknown architecture {name!r}; known: {sorted(ARCHITECTURES)}")
    module = importlib.import_module(ARCHITECTURES[name])
    if device is not None and torch.device(device).type == "cuda":
        from axlearn_b200.ops import cuda_ops

        cuda_ops.require_sources(module.KERNEL_SOURCES)
    tensors = read_safetensors(os.path.join(folder, "model.safetensors"))
    cfg = module.checkpoint_model_config(config, tensors).set(name="model", dtype=dtype)
    model = cfg.instantiate(parent=None)
    return LoadedModel(model, module.parameters(model, tensors, dtype=dtype, device=device), config, dtype)
