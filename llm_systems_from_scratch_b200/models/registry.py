"""Model registry: which class serves a configuration.

A configuration names its class under ``architecture``; the TransformerLM configurations that train.py writes
(model_config.json: the constructor's arguments) have no such key and select ``TransformerLM``."""
from __future__ import annotations

import json
import os

import torch

from .beledra import Beledra
from .genedra import Genedra
from .tedirax import Tedirax
from .transformer import TransformerLM
from .vilosun import Vilosun

MODELS = {"TransformerLM": TransformerLM, "Tedirax": Tedirax, "Beledra": Beledra, "Genedra": Genedra, "Vilosun": Vilosun}


def model_class(config: dict):
    name = config.get("architecture", "TransformerLM")
    if name not in MODELS:
        raise ValueError(f"unknown model architecture {name!r} (known: {', '.join(sorted(MODELS))})")
    return MODELS[name]


def vocabulary(config: dict) -> int:
    return config["vocab_size"] if "vocab_size" in config else config["vocab"]


def read_config(path: str) -> dict:
    """``path``: a configuration file, or a model folder with config.json (or model_config.json)."""
    if os.path.isdir(path):
        for name in ("config.json", "model_config.json"):
            if os.path.exists(os.path.join(path, name)):
                path = os.path.join(path, name)
                break
        else:
            raise FileNotFoundError(f"{path} has no config.json")
    with open(path) as f:
        return json.load(f)


def load_model(folder: str, dtype=torch.bfloat16, device="cuda"):
    """Load the model in ``folder`` (configuration and weights) for inference."""
    config = read_config(folder)
    cls = model_class(config)
    if hasattr(cls, "from_folder"):
        return cls.from_folder(folder, dtype, device)
    raise ValueError(f"{cls.__name__} is not loaded from a folder")


def build_model(config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda"):
    """A model of this configuration with random weights."""
    cls = model_class(config)
    if hasattr(cls, "random"):
        return cls.random(config, seed, dtype, device)
    torch.manual_seed(seed)
    with torch.device(device):
        return cls(**{k: v for k, v in config.items() if k != "architecture"}, use_custom_triton=True).eval()
