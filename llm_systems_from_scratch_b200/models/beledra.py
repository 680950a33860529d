"""Beledra: a decoder whose layers are listed one by one in the configuration, with norms behind the sublayers.

A layer is ``x <- x + norm1(mixer(x))`` and, unless its ``mlp`` is null, ``x <- x + norm2(ff(x))``: the sublayers read the
32-bit residual stream itself, and what they return is RMS-normed before it is added.  The mixers (``models/mixers.py``):

* ``mlstm``        matrix memory with exponential gates and a normaliser (``MatrixMemory``)
* ``attention``    grouped heads under a sliding window, normed queries and keys, a learned bias per distance bucket
* ``attention_2``  differential attention: two softmax maps over the same values, YaRN rotation, output gate; a layer with
  ``kv_from`` reads the keys and values of an earlier layer instead of having its own

config.json:
    vocab, width, norm.eps
    layers[i]       type, mixer {...}, mlp null or {kind: "dense", ff}
      mlstm         heads, dim, vdim, gate_cap
      attention     heads, kv_heads, dim, vdim, scale, mask: {size}, bias_max
      attention_2   heads, kv_heads, dim, vdim, scale, mask: {size}, diff, rot: {base, dims, scaling: {factor, original, fast,
                    slow}}, and optionally kv_from
Tensors: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, final.norm, head.

This class holds the configuration and the packed weights; caches, batches, scheduling and sampling belong to
``serving`` (``serving_backend`` connects the two).  Inference only.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field

import torch

from ..ops import mixer_ops as mo
from . import layered
from .layered import LayeredModel, need
from .mixers import GatedFeedForward, GroupedAttention, MatrixMemory


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class BeledraConfig:
    vocab: int
    width: int
    eps: float
    layers: list[LayerSpec] = field(default_factory=list)

    ATTENTION = ("heads", "kv_heads", "dim", "vdim", "scale", "mask")
    MIXER_KEYS = {"mlstm": ("heads", "dim", "vdim", "gate_cap"), "attention": (*ATTENTION, "bias_max"),
                  "attention_2": (*ATTENTION, "diff", "rot", "kv_from")}

    @classmethod
    def from_dict(cls, d: dict) -> "BeledraConfig":
        d = dict(d)
        d.pop("architecture", None)
        need(d, ("vocab", "width", "norm", "layers"), "config")
        need(d["norm"], ("eps",), "config norm")
        layers = []
        for i, entry in enumerate(d["layers"]):
            where = f"layer {i}"
            entry = {"mlp": None, **entry}
            need(entry, ("type", "mixer", "mlp"), where)
            if entry["type"] not in cls.MIXER_KEYS:
                raise ValueError(f"{where} has the unknown type {entry['type']!r}")
            m = dict(entry["mixer"])
            if entry["type"] == "attention_2":
                m.setdefault("kv_from", None)
            need(m, cls.MIXER_KEYS[entry["type"]], where + " mixer")
            if entry["type"] != "mlstm":
                need(m["mask"], ("size",), where + " mask")
                if m["mask"]["size"] < 1:
                    raise ValueError(f"{where} sees no key")
                if m["heads"] % m["kv_heads"]:
                    raise ValueError(f"{where}: the query heads must share the key heads evenly")
            if entry["type"] == "attention_2":
                m["rot"] = {"scaling": None, **m["rot"]}
                need(m["rot"], ("base", "dims", "scaling"), where + " rot")
                if m["rot"]["scaling"] is not None:
                    need(m["rot"]["scaling"], ("factor", "original", "fast", "slow"), where + " rot scaling")
                if m["kv_from"] is not None:
                    cls._check_source(i, m, layers, where)
            mlp = entry["mlp"]
            if mlp is not None:
                need(mlp, ("kind", "ff"), where + " mlp")
                if mlp["kind"] != "dense":
                    raise ValueError(f"{where} has the unknown feed-forward {mlp['kind']!r}")
            layers.append(LayerSpec(entry["type"], m, mlp))
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), layers)

    @staticmethod
    def _check_source(i: int, m: dict, layers: list, where: str):
        j = m["kv_from"]
        if not 0 <= j < i or layers[j].type != "attention_2" or layers[j].mixer["kv_from"] is not None:
            raise ValueError(f"{where} takes keys from layer {j}, which is no earlier layer with keys of its own")
        if any(m[k] != layers[j].mixer[k] for k in ("kv_heads", "dim", "vdim")):
            raise ValueError(f"{where} takes keys of other sizes from layer {j}")


class Layer:
    """One layer's packed weights."""

    def __init__(self, index: int, norm1, mixer, norm2, mlp):
        self.index, self.norm1, self.mixer, self.norm2, self.mlp = index, norm1, mixer, norm2, mlp


class Beledra(LayeredModel):
    KERNELS = ("grouped_attention.cu", "grouped_prefill.cu", "mlstm.cu")

    def __init__(self, config: dict, tensors, dtype=torch.bfloat16, device="cuda"):
        """``tensors[name]`` gives a tensor in its stored layout (a dict or a ``SafetensorsFile``)."""
        super().__init__(dtype, device)
        self.config = cfg = BeledraConfig.from_dict(config)
        self.embed = self.vector(tensors, "embed", cfg.vocab, cfg.width)
        for i, spec in enumerate(cfg.layers):
            pre = f"l{i}."
            norm2 = mlp = None
            if spec.mlp is not None:
                norm2 = self.vector(tensors, pre + "norm2", cfg.width)
                mlp = GatedFeedForward(lambda name: tensors[pre + "mlp." + name], cfg.width, spec.mlp["ff"], "relu", dtype, device)
            mixer = self._mixer(spec, lambda name: tensors[pre + "mix." + name])
            self.layers.append(Layer(i, self.vector(tensors, pre + "norm1", cfg.width), mixer, norm2, mlp))
        self.runs = self.layers
        self.final_norm = self.vector(tensors, "final.norm", cfg.width)
        self.head = mo.padded_weight(self.shaped(tensors, "head", cfg.vocab, cfg.width), dtype, device)
        self.vocab_size = cfg.vocab

    def _mixer(self, spec: LayerSpec, get):
        m, cfg = spec.mixer, self.config
        if spec.type == "mlstm":
            return MatrixMemory(get, cfg.width, m["heads"], m["dim"], m["vdim"], m["gate_cap"], cfg.eps, self.dtype, self.device)
        sizes = (get, cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["mask"]["size"], cfg.eps,
                 self.dtype, self.device)
        if spec.type == "attention":
            return GroupedAttention(*sizes, bias_max=m["bias_max"])
        rot = m["rot"]
        lam = self._difference(get, m["dim"], m["diff"])
        return GroupedAttention(*sizes, rope=self.rotary_table(rot["base"], rot["dims"], rot["scaling"]), rot_dims=rot["dims"],
                                difference=lam, out_scale=1.0 - m["diff"], gated=True, kv_from=m["kv_from"])

    @staticmethod
    def _difference(get, dim: int, diff: float) -> float:
        """Weight of the second map: exp(lq1 . lk1) - exp(lq2 . lk2) + diff, one number per layer."""
        dot = lambda a, b: float((get(a).double() * get(b).double()).sum())
        for name in ("lq1", "lk1", "lq2", "lk2"):
            if tuple(get(name).shape) != (dim,):
                raise ValueError(f"{name} has shape {tuple(get(name).shape)}, expected {(dim,)}")
        return math.exp(dot("lq1", "lk1")) - math.exp(dot("lq2", "lk2")) + diff

    @classmethod
    def random(cls, config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> "Beledra":
        """Random weights of the configuration's shapes (tests, benchmarks)."""
        return cls(config, RandomTensors(config, seed, device), dtype, device)

    # ------------------------------------------------------------------------------ serving hook
    def serving_backend(self):
        from ..serving.backends import PostNormLayers
        return PostNormLayers(self)


def RandomTensors(config: dict, seed: int = 0, device="cpu"):
    """Random weights on demand (``layered.RandomTensors``); the forget gates open, the vectors behind the weight of the second
    map are small."""
    def special(name, shape, kw):
        last = name.split(".mix.")[-1]
        if last in ("lq1", "lk1", "lq2", "lk2"):
            return (0.1 * torch.randn(shape, **kw)).to(torch.bfloat16)
        if last in ("i.b", "f.b"):
            return (torch.randn(shape, **kw) + (4.0 if last == "f.b" else -1.0)).to(torch.bfloat16)
        return None
    return layered.RandomTensors(tensor_shapes(BeledraConfig.from_dict(config)), seed, device, special)


BUCKETS = 32                      # rows of a distance table when nothing but the configuration is known


def tensor_shapes(cfg: BeledraConfig) -> dict[str, tuple[int, ...]]:
    """Name and shape of every tensor of a model of this configuration (distance tables: ``BUCKETS`` rows)."""
    w = cfg.width
    out = {"embed": (cfg.vocab, w)}
    for i, spec in enumerate(cfg.layers):
        m, pre = spec.mixer, f"l{i}."
        heads, dim, he = m["heads"], m["dim"], m["heads"] * m["vdim"]
        out[pre + "norm1"] = (w,)
        if spec.mlp is not None:
            out[pre + "norm2"] = (w,)
        if spec.type == "mlstm":
            hd = heads * dim
            mix = {"q": (hd, w), "k": (hd, w), "v": (he, w), "g": (he, w), "o": (w, he), "norm": (he,), "i": (heads, w),
                   "i.b": (heads,), "f": (heads, w), "f.b": (heads,)}
        else:
            maps, kv = (1 if spec.type == "attention" else 2), m["kv_heads"]
            mix = {"q": (heads * maps * dim, w), "q.norm": (dim,), "o": (w, he)}
            if m.get("kv_from") is None:
                mix.update({"k": (kv * maps * dim, w), "v": (kv * m["vdim"], w), "k.norm": (dim,)})
            if maps == 1:
                mix["rel"] = (BUCKETS, heads)
            else:
                mix.update({"lq1": (dim,), "lk1": (dim,), "lq2": (dim,), "lk2": (dim,), "g": (he, w)})
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if spec.mlp is not None:
            ff = spec.mlp["ff"]
            out.update({pre + "mlp.gate": (ff, w), pre + "mlp.up": (ff, w), pre + "mlp.down": (w, ff)})
    out["final.norm"] = (w,)
    out["head"] = (cfg.vocab, w)
    return out
