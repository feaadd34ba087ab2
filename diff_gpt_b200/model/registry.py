"""Which model class a checkpoint folder holds, and loading it.

A folder has `config.json`, whose "architecture" names the class, and `model.safetensors`.  A class is registered with
`from_config(config)` (a dict, as parsed) and `load_tensors({name: tensor})`.
"""

from __future__ import annotations

import json
import os

import torch

from ..weights import read_safetensors
from .delunex import Delunex
from .gpt import GPT, DeviceModel
from .kipolix import Kipolix

MODELS: dict[str, type[DeviceModel]] = {"GPT": GPT, "Delunex": Delunex, "Kipolix": Kipolix}


def model_class(config: dict) -> type[DeviceModel]:
    name = config.get("architecture")
    if name not in MODELS:
        raise ValueError(f"unknown architecture {name!r}; known: {', '.join(sorted(MODELS))}")
    return MODELS[name]


def load_model(folder: str, dtype: torch.dtype = torch.bfloat16, device: str | torch.device = "cuda") -> DeviceModel:
    with open(os.path.join(folder, "config.json")) as f:
        config = json.load(f)
    model = model_class(config).from_config(config).to(dtype)
    model.load_tensors(read_safetensors(os.path.join(folder, "model.safetensors")))
    return model.to(device).eval()
