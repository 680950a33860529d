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

from dataclasses import dataclass, field

import torch

from ..ops import mixer_ops as mo
from . import layered
from .layered import LayeredModel, need as _need
from .mixers import LatentAttention, Retention, TableExperts


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


class Tedirax(LayeredModel):
    KERNELS = ("flash_attn_fwd.cu", "latent_attention.cu", "latent_decode_tc.cu", "retention.cu")

    def __init__(self, config: dict, tensors, dtype=torch.bfloat16, device="cuda"):
        """``tensors[name]`` gives a tensor in its stored layout (a dict or a ``SafetensorsFile``)."""
        super().__init__(dtype, device)
        self.config = cfg = TediraxConfig.from_dict(config)
        self.embed = self.vector(tensors, "embed", cfg.vocab, cfg.width)
        for i, spec in enumerate(cfg.layers):
            pre = f"l{i}."
            norm = self.vector(tensors, pre + "norm1", cfg.width)
            mixer = self._mixer(spec, lambda name: tensors[pre + "mix." + name])
            experts = None
            if spec.mlp is not None:
                r = spec.mlp["router"]
                experts = TableExperts(lambda name: tensors[pre + "mlp." + name], cfg.width, spec.mlp["expert"]["ff"],
                                       r["experts"], r["top"], cfg.vocab, dtype, device)
            self.layers.append(Layer(i, norm, mixer, experts))
        self.runs = [self.layers[i] for i in cfg.runs()]
        self.final_norm = self.vector(tensors, "final.norm", cfg.width)
        self.head = mo.padded_weight(self.shaped(tensors, "head", cfg.vocab, cfg.width), dtype, device)
        self.vocab_size = cfg.vocab

    def _mixer(self, spec: LayerSpec, get):
        m, cfg = spec.mixer, self.config
        if spec.type == "latent_attention":
            return LatentAttention(get, cfg.width, m["heads"], m["dim"], m["vdim"], m["q_rank"], m["kv_rank"], m["scale"],
                                   m["mask"]["size"], cfg.eps, self.dtype, self.device)
        rot = m["rot"]
        return Retention(get, cfg.width, m["heads"], m["dim"], m["vdim"], m["decay"], rot["dims"], cfg.eps,
                         self.rotary_table(rot["base"], rot["dims"]), self.dtype, self.device)

    @classmethod
    def random(cls, config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> "Tedirax":
        """Random weights of the configuration's shapes (tests, benchmarks)."""
        return cls(config, RandomTensors(config, seed, device), dtype, device)

    # ------------------------------------------------------------------------------ serving hook
    def serving_backend(self):
        from ..serving.backends import ParallelLayers
        return ParallelLayers(self)


def RandomTensors(config: dict, seed: int = 0, device="cpu"):
    """Random weights on demand (``layered.RandomTensors``); the experts of a token are drawn without repetition."""
    cfg = TediraxConfig.from_dict(config)

    def table(name, shape, kw):
        if name.endswith(".table"):
            experts = cfg.layers[int(name[1:].split(".")[0])].mlp["router"]["experts"]
            return torch.rand((shape[0], experts), **kw).argsort(1)[:, :shape[1]].to(torch.int32)
        return None
    return layered.RandomTensors(tensor_shapes(cfg), seed, device, table)


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
