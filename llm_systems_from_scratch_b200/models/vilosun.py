"""Vilosun: a decoder whose layers are listed one by one in the configuration, with gated sublayers between norms.

A layer is ``x <- x + norm1b(mixer(h) * sigmoid(W_rg1 h + b))`` with ``h = norm1(x)`` and, unless its ``mlp`` is null, the same with norm2,
norm2b, rg2 and its experts.  Norms are RMS norms of equal consecutive parts of the width; the embedding is scaled and joined by a row for the
pair (previous token, token); logits are multiplied by a number.  The mixers (``models/mixers.py``):

* ``attention``  grouped heads inside chunks of positions, biases and a short convolution on q, k and v, a factor and a distance slope per head,
  values mixed with those of the first layer that mixes, a gate per head
* ``delta``      the gated delta rule with a short convolution on q, k and v

and the feed-forward: gated experts chosen by a router.

config.json:
    vocab, width, norm {eps, groups}, embedding {scale, bigram {buckets, mul_prev, mul_cur}}, logit_scale
    layers[i]       type, mixer {...}, mlp null or {kind: "moe", expert: {ff}, router: {experts, top}}
      attention     heads, kv_heads, dim, vdim, scale, conv, mask {size}, v_mix
      delta         heads, kv_heads, dim, vdim, conv
Tensors: embed, bigram, l<i>.norm1, .norm1b, .rg1, .rg1.b, l<i>.mix.*, with a feed-forward l<i>.norm2, .norm2b, .rg2, .rg2.b and l<i>.mlp.*,
final.norm, head.

This class holds the configuration and the packed weights; caches, batches, scheduling and sampling belong to
``serving`` (``serving_backend`` connects the two).  Inference only.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops import mixer_ops as mo
from . import layered
from .layered import LayeredModel, need
from .mixers import DeltaRule, GroupedAttention, RoutedExperts


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class VilosunConfig:
    vocab: int
    width: int
    eps: float
    groups: int
    embed_scale: float
    buckets: int
    mul_prev: int
    mul_cur: int
    logit_scale: float
    layers: list[LayerSpec] = field(default_factory=list)

    MIXER_KEYS = {"attention": ("heads", "kv_heads", "dim", "vdim", "scale", "conv", "mask", "v_mix"),
                  "delta": ("heads", "kv_heads", "dim", "vdim", "conv")}

    @classmethod
    def from_dict(cls, d: dict) -> "VilosunConfig":
        d = dict(d)
        d.pop("architecture", None)
        need(d, ("vocab", "width", "norm", "embedding", "logit_scale", "layers"), "config")
        need(d["norm"], ("eps", "groups"), "config norm")
        need(d["embedding"], ("scale", "bigram"), "config embedding")
        pairs = d["embedding"]["bigram"]
        need(pairs, ("buckets", "mul_prev", "mul_cur"), "config bigram")
        if pairs["buckets"] < 1:
            raise ValueError("the embedding of pairs has no rows")
        if d["norm"]["groups"] < 1 or d["width"] % d["norm"]["groups"]:
            raise ValueError(f"{d['width']} columns do not make {d['norm']['groups']} equal groups")
        layers = []
        for i, entry in enumerate(d["layers"]):
            where = f"layer {i}"
            entry = {"mlp": None, **entry}
            need(entry, ("type", "mixer", "mlp"), where)
            if entry["type"] not in cls.MIXER_KEYS:
                raise ValueError(f"{where} has the unknown type {entry['type']!r}")
            m = dict(entry["mixer"])
            if entry["type"] == "attention":
                m.setdefault("v_mix", False)
            need(m, cls.MIXER_KEYS[entry["type"]], where + " mixer")
            if m["heads"] % m["kv_heads"]:
                raise ValueError(f"{where}: the heads must share the key heads evenly")
            if entry["type"] == "attention":
                need(m["mask"], ("size",), where + " mask")
                if m["mask"]["size"] < 1:
                    raise ValueError(f"{where} sees no key")
            layers.append(LayerSpec(entry["type"], m, cls._check_mlp(entry["mlp"], where + " mlp")))
        c = cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), int(d["norm"]["groups"]), float(d["embedding"]["scale"]),
                int(pairs["buckets"]), int(pairs["mul_prev"]), int(pairs["mul_cur"]), float(d["logit_scale"]), layers)
        first = c.first_values
        for i, spec in enumerate(layers):
            if spec.type == "attention" and spec.mixer["v_mix"] and any(spec.mixer[k] != layers[first].mixer[k] for k in ("kv_heads", "vdim")):
                raise ValueError(f"layer {i} mixes its values with others of another size")
        return c

    @staticmethod
    def _check_mlp(mlp, where: str):
        if mlp is None:
            return None
        if mlp.get("kind") != "moe":
            raise ValueError(f"{where} has the unknown kind {mlp.get('kind')!r}")
        need(mlp, ("kind", "expert", "router"), where)
        need(mlp["expert"], ("ff",), where + " expert")
        need(mlp["router"], ("experts", "top"), where + " router")
        r = mlp["router"]
        if not 0 < r["top"] <= r["experts"]:
            raise ValueError(f"{where}: {r['top']} of {r['experts']} experts cannot be chosen")
        return mlp

    @property
    def first_values(self) -> int | None:
        """The first layer that mixes values: the others mix theirs with its."""
        return next((i for i, s in enumerate(self.layers) if s.type == "attention" and s.mixer["v_mix"]), None)


class Layer:
    """One layer's packed weights."""

    def __init__(self, index: int, norm1, mixer, norm1b, norm2, mlp, norm2b):
        self.index, self.norm1, self.mixer, self.norm1b = index, norm1, mixer, norm1b
        self.norm2, self.mlp, self.norm2b = norm2, mlp, norm2b


class Vilosun(LayeredModel):
    KERNELS = ("grouped_attention.cu", "grouped_prefill.cu", "moe_route.cu", "short_conv.cu", "delta.cu", "group_norm.cu")

    def __init__(self, config: dict, tensors, dtype=torch.bfloat16, device="cuda"):
        """``tensors[name]`` gives a tensor in its stored layout (a dict or a ``SafetensorsFile``)."""
        super().__init__(dtype, device)
        self.config = cfg = VilosunConfig.from_dict(config)
        self.embed = self.vector(tensors, "embed", cfg.vocab, cfg.width)
        self.bigram = self.vector(tensors, "bigram", cfg.buckets + 1, cfg.width)
        for i, spec in enumerate(cfg.layers):
            norm = lambda name: self.vector(tensors, f"l{i}.{name}", cfg.width)
            gate = lambda name: (self.shaped(tensors, f"l{i}.{name}", cfg.width, cfg.width), self.shaped(tensors, f"l{i}.{name}.b", cfg.width))
            mixer = self._mixer(i, spec, lambda name: tensors[f"l{i}.mix.{name}"], gate("rg1"))
            norm2 = mlp = norm2b = None
            if spec.mlp is not None:
                r = spec.mlp["router"]
                mlp = RoutedExperts(lambda name: tensors[f"l{i}.mlp.{name}"], cfg.width, spec.mlp["expert"]["ff"], r["experts"], r["top"], 0, None,
                                    dtype, device, gated=True, choice="logits", out_gate=gate("rg2"))
                norm2, norm2b = norm("norm2"), norm("norm2b")
            self.layers.append(Layer(i, norm("norm1"), mixer, norm("norm1b"), norm2, mlp, norm2b))
        self.runs = self.layers
        self.final_norm = self.vector(tensors, "final.norm", cfg.width)
        self.head = mo.padded_weight(self.shaped(tensors, "head", cfg.vocab, cfg.width), dtype, device)
        self.vocab_size = cfg.vocab

    def _mixer(self, index: int, spec: LayerSpec, get, out_gate):
        m, cfg = spec.mixer, self.config
        sizes = (get, cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"])
        if spec.type == "delta":
            return DeltaRule(*sizes, m["conv"], cfg.eps, self.dtype, self.device, out_gate=out_gate)
        first = cfg.first_values
        return GroupedAttention(*sizes, m["scale"], m["mask"]["size"], cfg.eps, self.dtype, self.device, biased="inputs", norm=None, chunked=True,
                                slopes=[2.0 ** (-8.0 * (h + 1) / m["heads"]) for h in range(m["heads"])], conv=m["conv"], temp=True,
                                mix_from=first if m["v_mix"] and index != first else None, gated="heads", out_gate=out_gate)

    @classmethod
    def random(cls, config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> "Vilosun":
        """Random weights of the configuration's shapes (tests, benchmarks)."""
        return cls(config, RandomTensors(config, seed, device), dtype, device)

    # ------------------------------------------------------------------------------ serving hook
    def serving_backend(self):
        from ..serving.backends import SandwichLayers
        return SandwichLayers(self)


def RandomTensors(config: dict, seed: int = 0, device="cpu"):
    """Random weights on demand (``layered.RandomTensors``); biases are small, decays slow, filters weigh the current token most."""
    def special(name, shape, kw):
        last = name.split(".")[-1]
        rnd = lambda mean, std: (mean + std * torch.randn(shape, **kw)).to(torch.bfloat16)
        if name == "bigram":
            return rnd(0.0, 1.0)
        if last == "conv":
            t = rnd(0.0, 0.3)
            t[:, -1] += 1.0
            return t
        return {"b": lambda: rnd(0.0, 0.1), "A_log": lambda: rnd(-1.0, 0.5), "dt_bias": lambda: rnd(-2.0, 0.5), "vmix": lambda: rnd(0.5, 0.1)}[last]() \
            if (last in ("A_log", "dt_bias", "vmix") or (last == "b" and len(shape) == 1)) else None
    return layered.RandomTensors(tensor_shapes(VilosunConfig.from_dict(config)), seed, device, special)


def tensor_shapes(cfg: VilosunConfig) -> dict[str, tuple[int, ...]]:
    """Name and shape of every tensor of a model of this configuration."""
    w = cfg.width
    out = {"embed": (cfg.vocab, w), "bigram": (cfg.buckets + 1, w)}
    for i, spec in enumerate(cfg.layers):
        m, mlp, pre = spec.mixer, spec.mlp, f"l{i}."
        heads, kv, dim, he, taps = m["heads"], m["kv_heads"], m["dim"], m["heads"] * m["vdim"], m["conv"]
        out.update({pre + "norm1": (w,), pre + "norm1b": (w,), pre + "rg1": (w, w), pre + "rg1.b": (w,)})
        if spec.type == "attention":
            rows = {"q": heads * dim, "k": kv * dim, "v": kv * m["vdim"]}
            mix = {"temp": (heads,), "g": (heads, w), "o": (w, he)}
            mix.update({name + ".b": (n,) for name, n in rows.items()})
            if m["v_mix"]:
                mix["vmix"] = ()
        else:
            rows = {"q": kv * dim, "k": kv * dim, "v": he}
            mix = {"a": (heads, w), "b": (heads, w), "A_log": (heads,), "dt_bias": (heads,), "norm": (m["vdim"],), "g": (he, w), "o": (w, he)}
        for name, n in rows.items():
            mix.update({name: (n, w), name + ".conv": (n, taps)})
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if mlp is None:
            continue
        f, r = mlp["expert"]["ff"], mlp["router"]
        ff = {f"e{e}.{k}": v for e in range(r["experts"]) for k, v in (("gate", (f, w)), ("up", (f, w)), ("down", (w, f)))}
        ff.update({"router": (r["experts"], w), "router.b": (r["experts"],)})
        out.update({pre + "norm2": (w,), pre + "norm2b": (w,), pre + "rg2": (w, w), pre + "rg2.b": (w,)})
        out.update({pre + "mlp." + k: v for k, v in ff.items()})
    out["final.norm"] = (w,)
    out["head"] = (cfg.vocab, w)
    return out
