"""Tedirax: a decoder whose layers are listed one by one in the configuration.

Every layer is parallel - one RMS norm, and mixer and feed-forward both read its output:
``x <- x + (mixer(h) + ff(h))`` - with its own mixer (``retention`` or ``latent_attention``, ``models/mixers.py``), its own
sizes and an optional mixture of table-chosen experts.  A range of layers can be run several times in a row with the
same weights; every pass keeps a cache or state of its own.

config.json:
    vocab, width, norm.eps
    loop            null, or start / stop / times: layers start .. stop - 1 run ``times`` times
    layers[i]       type, mixer {...}, mlp null or {kind: "moe", expert: {ff}, router: {experts, top}}
      retention         heads, dim, vdim, decay (one per head), rot: {base, dims}
      latent_attention  heads, dim, vdim, q_rank, kv_rank, scale, mask: {size}
Tensors: embed, l<i>.norm1, l<i>.mix.*, l<i>.mlp.*, final.norm, head.

This class holds the configuration and the packed weights; caches, batches, scheduling and sampling belong to
``serving`` (``serving_backend`` connects the two).  Inference only.
"""
from __future__ import annotations

import json
import os
import warnings
from dataclasses import dataclass, field

import torch

from ..ops import mixer_ops as mo
from ..utils.safetensors import SafetensorsFile
from .mixers import LatentAttention, Retention, RotaryTable, TableExperts


def _need(d: dict, keys, where: str):
    missing = [k for k in keys if k not in d]
    if missing:
        raise ValueError(f"{where} lacks {', '.join(missing)}")
    extra = [k for k in d if k not in keys]
    if extra:
        warnings.warn(f"{where} has settings this design does not know: {', '.join(extra)}", stacklevel=3)


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class TediraxConfig:
    vocab: int
    width: int
    eps: float
    layers: list[LayerSpec] = field(default_factory=list)
    loop: tuple[int, int, int] | None = None        # start, stop, times

    MIXER_KEYS = {"retention": ("heads", "dim", "vdim", "decay", "rot"),
                  "latent_attention": ("heads", "dim", "vdim", "q_rank", "kv_rank", "scale", "mask")}

    @classmethod
    def from_dict(cls, d: dict) -> "TediraxConfig":
        d = dict(d)
        d.pop("architecture", None)
        d.setdefault("loop", None)
        _need(d, ("vocab", "width", "norm", "layers", "loop"), "config")
        _need(d["norm"], ("eps",), "config norm")
        layers = []
        for i, entry in enumerate(d["layers"]):
            where = f"layer {i}"
            entry = dict(entry)
            entry.setdefault("mlp", None)
            _need(entry, ("type", "mixer", "mlp"), where)
            if entry["type"] not in cls.MIXER_KEYS:
                raise ValueError(f"{where} has the unknown type {entry['type']!r}")
            _need(entry["mixer"], cls.MIXER_KEYS[entry["type"]], where + " mixer")
            if entry["type"] == "retention":
                _need(entry["mixer"]["rot"], ("base", "dims"), where + " rot")
            else:
                _need(entry["mixer"]["mask"], ("size",), where + " mask")
            mlp = entry["mlp"]
            if mlp is not None:
                _need(mlp, ("kind", "expert", "router"), where + " mlp")
                if mlp["kind"] != "moe":
                    raise ValueError(f"{where} has the unknown feed-forward {mlp['kind']!r}")
                _need(mlp["expert"], ("ff",), where + " expert")
                _need(mlp["router"], ("experts", "top"), where + " router")
            layers.append(LayerSpec(entry["type"], entry["mixer"], mlp))
        loop = None
        if d["loop"] is not None:
            _need(d["loop"], ("start", "stop", "times"), "config loop")
            loop = (int(d["loop"]["start"]), int(d["loop"]["stop"]), int(d["loop"]["times"]))
            if not (0 <= loop[0] <= loop[1] <= len(layers)) or loop[2] < 0:
                raise ValueError("config loop does not fit the layers")
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers, loop)

    def runs(self) -> list[int]:
        """Layer index of every layer run, in order."""
        n = len(self.layers)
        if self.loop is None:
            return list(range(n))
        a, b, times = self.loop
        return [*range(a), *list(range(a, b)) * times, *range(b, n)]


class Layer:
    """One layer's packed weights; ``run`` indices that share it share them too."""

    def __init__(self, index: int, norm, mixer, experts):
        self.index, self.norm, self.mixer, self.experts = index, norm, mixer, experts


class Tedirax:
    GPU_DTYPES = (torch.bfloat16, torch.float32)
    DEFAULT_CONTEXT = 4096            # positions an engine serves unless it is told otherwise; the design has no limit

    def __init__(self, config: dict, tensors, dtype=torch.bfloat16, device="cuda"):
        """``tensors[name]`` gives a tensor in its stored layout (a dict or a ``SafetensorsFile``)."""
        if dtype not in self.GPU_DTYPES:
            raise ValueError("Tedirax runs in bfloat16 or float32")
        self.config = cfg = TediraxConfig.from_dict(config)
        self.dtype, self.device = dtype, torch.device(device)
        take = lambda name, *shape: self._shaped(tensors, name, shape)
        self.embed = take("embed", cfg.vocab, cfg.width).to(device=device, dtype=dtype).contiguous()
        self.rotary: dict[tuple, RotaryTable] = {}
        self.layers = []
        for i, spec in enumerate(cfg.layers):
            pre = f"l{i}."
            norm = take(pre + "norm1", cfg.width).to(device=device, dtype=dtype).contiguous()
            mixer = self._mixer(spec, lambda name: tensors[pre + "mix." + name])
            experts = None
            if spec.mlp is not None:
                r = spec.mlp["router"]
                experts = TableExperts(lambda name: tensors[pre + "mlp." + name], cfg.width, spec.mlp["expert"]["ff"],
                                       r["experts"], r["top"], cfg.vocab, dtype, device)
            self.layers.append(Layer(i, norm, mixer, experts))
        self.runs = [self.layers[i] for i in cfg.runs()]
        self.final_norm = take("final.norm", cfg.width).to(device=device, dtype=dtype).contiguous()
        self.head = mo.padded_weight(take("head", cfg.vocab, cfg.width), dtype, device)
        self.vocab_size = cfg.vocab
        self._engine = None

    @staticmethod
    def _shaped(tensors, name, shape):
        t = tensors[name]
        if tuple(t.shape) != shape:
            raise ValueError(f"{name} has shape {tuple(t.shape)}, expected {shape}")
        return t

    def _mixer(self, spec: LayerSpec, get):
        m, cfg = spec.mixer, self.config
        if spec.type == "latent_attention":
            return LatentAttention(get, cfg.width, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"],
                                   m["mask"]["size"], cfg.eps, self.dtype, self.device)
        dims = m["rot"]["dims"]
        rope = None
        if dims:
            rope = self.rotary.setdefault((m["rot"]["base"], dims), RotaryTable(m["rot"]["base"], dims, self.device))
        return Retention(get, cfg.width, m["heads"], m["dim"], m["vdim"], m["decay"], dims, cfg.eps, rope, self.dtype, self.device)

    # ---------------------------------------------------------------------------------- loading
    @classmethod
    def from_folder(cls, folder: str, dtype=torch.bfloat16, device="cuda") -> "Tedirax":
        """``folder``: config.json and model.safetensors."""
        with open(os.path.join(folder, "config.json")) as f:
            config = json.load(f)
        return cls(config, SafetensorsFile(os.path.join(folder, "model.safetensors")), dtype, device)

    @classmethod
    def random(cls, config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> "Tedirax":
        """Random weights of the configuration's shapes (tests, benchmarks)."""
        return cls(config, RandomTensors(config, seed, device), dtype, device)

    def eval(self):
        return self

    # ------------------------------------------------------------------------------ serving hook
    def serving_backend(self):
        from ..serving.backends import LayeredBackend
        return LayeredBackend(self)

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
    """Weights made on demand: normal with variance 1 / fan-in, norms around one, experts drawn without repetition."""

    def __init__(self, config: dict, seed: int = 0, device="cpu"):
        self.cfg, self.seed, self.device = TediraxConfig.from_dict(config), seed, torch.device(device)
        self.shapes = tensor_shapes(self.cfg)
        self._order = {name: i for i, name in enumerate(self.shapes)}

    def keys(self):
        return self.shapes.keys()

    def __getitem__(self, name: str):
        shape = self.shapes[name]
        g = torch.Generator(self.device).manual_seed(self.seed * 1000003 + self._order[name])
        kw = {"generator": g, "device": self.device}
        if name.endswith(".table"):
            experts = self.cfg.layers[int(name[1:].split(".")[0])].mlp["router"]["experts"]
            return torch.rand((shape[0], experts), **kw).argsort(1)[:, :shape[1]].to(torch.int32)
        if len(shape) == 1:
            return (1.0 + 0.1 * torch.randn(shape, **kw)).to(torch.bfloat16)
        std = 1.0 if name == "embed" else shape[1] ** -0.5
        return (std * torch.randn(shape, **kw)).to(torch.bfloat16)


def tensor_shapes(cfg: TediraxConfig) -> dict[str, tuple[int, ...]]:
    """Name and shape of every tensor of a model of this configuration."""
    w = cfg.width
    out = {"embed": (cfg.vocab, w)}
    for i, spec in enumerate(cfg.layers):
        m, pre = spec.mixer, f"l{i}."
        out[pre + "norm1"] = (w,)
        hd, he = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        if spec.type == "retention":
            mix = {"q": (hd, w), "k": (hd, w), "v": (he, w), "g": (he, w), "o": (w, he)}
        else:
            qr, kr = m["q_rank"], m["kv_rank"]
            mix = {"dq": (qr, w), "dq.norm": (qr,), "uq": (hd, qr), "dkv": (kr, w), "dkv.norm": (kr,), "uk": (hd, kr),
                   "uv": (he, kr), "g": (he, w), "o": (w, he)}
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if spec.mlp is not None:
            ff, r = spec.mlp["expert"]["ff"], spec.mlp["router"]
            for e in range(r["experts"]):
                out.update({f"{pre}mlp.e{e}.gate": (ff, w), f"{pre}mlp.e{e}.up": (ff, w), f"{pre}mlp.e{e}.down": (w, ff)})
            out[pre + "mlp.table"] = (cfg.vocab, r["top"])
    out["final.norm"] = (w,)
    out["head"] = (cfg.vocab, w)
    return out
