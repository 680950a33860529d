"""What models made of listed layers have in common (``tedirax.py``, ``beledra.py``, ``genedra.py``, ``vilosun.py``): configuration checks,
loading from a folder, random weights, generation through the serving engine.

A subclass reads its configuration, packs its weights into ``layers`` / ``runs`` (objects with a ``mixer`` from ``mixers.py``
among others) and names the serving backend that knows its order of sublayers; caches, batches, scheduling and sampling
belong to ``serving``.  Inference only."""
from __future__ import annotations

import json
import os
import warnings

import torch

from ..utils.safetensors import SafetensorsFile
from .mixers import RotaryTable


def need(d: dict, keys, where: str):
    """Check that ``d`` has these settings; others are ignored with a warning."""
    missing = [k for k in keys if k not in d]
    if missing:
        raise ValueError(f"{where} lacks {', '.join(missing)}")
    extra = [k for k in d if k not in keys]
    if extra:
        warnings.warn(f"{where} has settings this design does not know: {', '.join(extra)}", stacklevel=3)


class LayeredModel:
    GPU_DTYPES = (torch.bfloat16, torch.float32)
    KERNELS = None                    # CUDA sources of its mixers (build_ext.MIXERS); None: all of them
    DEFAULT_CONTEXT = 4096            # positions an engine serves unless it is told otherwise; the designs have no limit

    def __init__(self, dtype, device):
        if dtype not in self.GPU_DTYPES:
            raise ValueError(f"{type(self).__name__} runs in bfloat16 or float32")
        self.dtype, self.device = dtype, torch.device(device)
        self.rotary: dict[tuple, RotaryTable] = {}
        self.layers, self.runs = [], []
        self._engine = None

    # ---------------------------------------------------------------------------------- loading
    @staticmethod
    def shaped(tensors, name, *shape):
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name} has shape {tuple(t.shape)}, expected {shape}")
        return t

    def vector(self, tensors, name, *shape):
        """A tensor the kernels read as it is stored, in the model's type."""
        return self.shaped(tensors, name, *shape).to(device=self.device, dtype=self.dtype).contiguous()

    def rotary_table(self, base, dims, scaling=None):
        """The angle table of this rotation, shared by the layers that use it (None without rotated dimensions)."""
        if not dims:
            return None
        key = (base, dims, None if scaling is None else tuple(sorted(scaling.items())))
        if key not in self.rotary:
            self.rotary[key] = RotaryTable(base, dims, self.device, scaling)
        return self.rotary[key]

    @classmethod
    def from_folder(cls, folder: str, dtype=torch.bfloat16, device="cuda"):
        """``folder``: config.json and model.safetensors."""
        with open(os.path.join(folder, "config.json")) as f:
            config = json.load(f)
        return cls(config, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype, device)

    def eval(self):
        return self

    # ------------------------------------------------------------------------------ generation
    @torch.no_grad()
    def generate(self, prompt_ids, max_new_tokens: int, temperature: float = 1.0, top_k: int | None = None,
                 eos_token_id: int | None = None):
        """Up to ``max_new_tokens`` ids after the prompt, shape (1, n), through the serving engine; the stop token is not
        returned (as in ``TransformerLM.generate``)."""
        from ..serving import ServingEngine
        ids = prompt_ids.reshape(-1).tolist()
        total = len(ids) + max_new_tokens
        if self._engine is None or self._engine.max_context < total:
            ctx = -(-total // 256) * 256
            self._engine = ServingEngine(self, num_pages=-(-ctx // 64), page_size=64, max_batch=1, max_context=ctx,
                                         use_cuda_graphs=False)
        out = self._engine.generate([ids], max_new_tokens, eos_token_id, temperature, top_k)[0]
        if eos_token_id is not None and out and out[-1] == eos_token_id:
            out = out[:-1]
        return torch.tensor([out], dtype=torch.long, device=self.device).reshape(1, -1)


class RandomTensors:
    """Weights made on demand from ``shapes`` (name -> shape): matrices normal with variance 1 / fan-in, vectors around one;
    ``special(name, shape, generator keywords)`` may make others."""

    def __init__(self, shapes: dict, seed: int = 0, device="cpu", special=None):
        self.shapes, self.seed, self.device, self.special = shapes, seed, torch.device(device), special
        self._order = {name: i for i, name in enumerate(shapes)}

    def keys(self):
        return self.shapes.keys()

    def __getitem__(self, name: str):
        shape = self.shapes[name]
        kw = {"generator": torch.Generator(self.device).manual_seed(self.seed * 1000003 + self._order[name]), "device": self.device}
        t = self.special(name, shape, kw) if self.special is not None else None
        if t is not None:
            return t
        if len(shape) <= 1:
            return (1.0 + 0.1 * torch.randn(shape, **kw)).to(torch.bfloat16)
        std = 1.0 if name == "embed" else shape[1] ** -0.5
        return (std * torch.randn(shape, **kw)).to(torch.bfloat16)
