"""Genedra: a decoder whose layers are listed one by one in the configuration, with a norm in front of every sublayer.

A layer is ``x <- x + m mixer(norm1(x))`` and, unless its ``mlp`` is null, ``x <- x + m ff(norm2(x))``, m one number for the whole
model; norm weights are stored as their distance from one; the embedding is scaled, the logits are capped softly.  The mixers
(``models/mixers.py``):

* ``latent_attention``  keys and values from one cached latent per token, a rotated key part shared by all heads, a gate per head; a
  layer with ``kv_from`` reads the cache of an earlier one
* ``attention``         grouped heads with biases, one norm over all queries (and keys), partly rotated, capped scores, a sliding window
  beside the first tokens, a sink per head

and the feed-forwards: a dense SwiGLU, or experts chosen by a router (some of its outputs are the input itself) beside a gated
shared one.

config.json:
    vocab, width, norm.eps, embedding.scale, residual_mult, logit_softcap
    layers[i]           type, mixer {...}, mlp null or {kind: "dense", ff} or {kind: "moe", expert: {ff}, router: {experts, top,
                        identity}, shared: {ff}}
      latent_attention  heads, dim, vdim, kv_rank, rot_dim, scale, rot: {base, dims}, and optionally kv_from
      attention         heads, kv_heads, dim, vdim, scale, softcap, mask: {size, keep_first}, rot: {base, dims, scaling: {factor}}
Tensors: embed, l<i>.norm1, l<i>.norm2, l<i>.mix.*, l<i>.mlp.*, final.norm, head.

This class holds the configuration and the packed weights; caches, batches, scheduling and sampling belong to
``serving`` (``serving_backend`` connects the two).  Inference only.
"""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops import mixer_ops as mo
from . import layered
from .layered import LayeredModel, need
from .mixers import GatedFeedForward, GroupedAttention, LatentAttention, RoutedExperts


@dataclass
class LayerSpec:
    type: str
    mixer: dict
    mlp: dict | None


@dataclass
class GenedraConfig:
    vocab: int
    width: int
    eps: float
    embed_scale: float
    gain: float
    logit_softcap: float
    layers: list[LayerSpec] = field(default_factory=list)

    MIXER_KEYS = {"latent_attention": ("heads", "dim", "vdim", "kv_rank", "rot_dim", "scale", "rot", "kv_from"),
                  "attention": ("heads", "kv_heads", "dim", "vdim", "scale", "softcap", "mask", "rot")}

    @classmethod
    def from_dict(cls, d: dict) -> "GenedraConfig":
        d = dict(d)
        d.pop("architecture", None)
        need(d, ("vocab", "width", "norm", "embedding", "residual_mult", "logit_softcap", "layers"), "config")
        need(d["norm"], ("eps",), "config norm")
        need(d["embedding"], ("scale",), "config embedding")
        if d["logit_softcap"] <= 0:
            raise ValueError("the cap of the logits must be positive")
        layers = []
        for i, entry in enumerate(d["layers"]):
            where = f"layer {i}"
            entry = {"mlp": None, **entry}
            need(entry, ("type", "mixer", "mlp"), where)
            if entry["type"] not in cls.MIXER_KEYS:
                raise ValueError(f"{where} has the unknown type {entry['type']!r}")
            m = dict(entry["mixer"])
            if entry["type"] == "latent_attention":
                cls._check_latent(i, m, layers, where)
            else:
                cls._check_attention(m, where)
            layers.append(LayerSpec(entry["type"], m, cls._check_mlp(entry["mlp"], where)))
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["residual_mult"]),
                   float(d["logit_softcap"]), layers)

    @classmethod
    def _check_latent(cls, i: int, m: dict, layers: list, where: str):
        m.setdefault("kv_from", None)
        need(m, cls.MIXER_KEYS["latent_attention"], where + " mixer")
        need(m["rot"], ("base", "dims"), where + " rot")
        if m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2:
            raise ValueError(f"{where} rotates all of its rot_dim dimensions, pair by pair")
        j = m["kv_from"]
        if j is None:
            return
        if not 0 <= j < i or layers[j].type != "latent_attention" or layers[j].mixer["kv_from"] is not None:
            raise ValueError(f"{where} takes latents from layer {j}, which is no earlier layer with latents of its own")
        if any(m[k] != layers[j].mixer[k] for k in ("kv_rank", "rot_dim", "rot")):
            raise ValueError(f"{where} takes latents of another size or rotation from layer {j}")

    @classmethod
    def _check_attention(cls, m: dict, where: str):
        need(m, cls.MIXER_KEYS["attention"], where + " mixer")
        m["mask"], m["rot"] = {"keep_first": 0, **m["mask"]}, {"scaling": None, **m["rot"]}
        need(m["mask"], ("size", "keep_first"), where + " mask")
        need(m["rot"], ("base", "dims", "scaling"), where + " rot")
        if m["rot"]["scaling"] is not None:
            need(m["rot"]["scaling"], ("factor",), where + " rot scaling")
        if m["mask"]["size"] < 1 or m["mask"]["keep_first"] < 0:
            raise ValueError(f"{where} sees no key")
        if m["heads"] % m["kv_heads"]:
            raise ValueError(f"{where}: the query heads must share the key heads evenly")
        if m["softcap"] <= 0:
            raise ValueError(f"{where}: the cap of the scores must be positive")

    @staticmethod
    def _check_mlp(mlp, where: str):
        if mlp is None:
            return None
        where += " mlp"
        if mlp.get("kind") == "dense":
            need(mlp, ("kind", "ff"), where)
            return mlp
        if mlp.get("kind") != "moe":
            raise ValueError(f"{where} has the unknown kind {mlp.get('kind')!r}")
        mlp = {"shared": None, **mlp}
        need(mlp, ("kind", "expert", "router", "shared"), where)
        mlp["router"] = r = {"identity": 0, **mlp["router"]}
        need(r, ("experts", "top", "identity"), where + " router")
        need(mlp["expert"], ("ff",), where + " expert")
        if mlp["shared"] is not None:
            need(mlp["shared"], ("ff",), where + " shared")
        if not 0 < r["top"] <= r["experts"] + r["identity"]:
            raise ValueError(f"{where}: {r['top']} of {r['experts'] + r['identity']} outputs cannot be chosen")
        return mlp


class Layer:
    """One layer's packed weights."""

    def __init__(self, index: int, norm1, mixer, norm2, mlp):
        self.index, self.norm1, self.mixer, self.norm2, self.mlp = index, norm1, mixer, norm2, mlp
        self.routed = isinstance(mlp, RoutedExperts)


class Genedra(LayeredModel):
    KERNELS = ("flash_attn_fwd.cu", "latent_attention.cu", "latent_decode_tc.cu", "grouped_attention.cu", "grouped_prefill.cu",
               "moe_route.cu")

    def __init__(self, config: dict, tensors, dtype=torch.bfloat16, device="cuda"):
        """``tensors[name]`` gives a tensor in its stored layout (a dict or a ``SafetensorsFile``)."""
        super().__init__(dtype, device)
        self.config = cfg = GenedraConfig.from_dict(config)
        self.embed = self.vector(tensors, "embed", cfg.vocab, cfg.width)
        for i, spec in enumerate(cfg.layers):
            pre = f"l{i}."
            norm2 = mlp = None
            if spec.mlp is not None:
                norm2 = self.vector(tensors, pre + "norm2", cfg.width)
                mlp = self._mlp(spec.mlp, lambda name: tensors[pre + "mlp." + name])
            mixer = self._mixer(spec, lambda name: tensors[pre + "mix." + name])
            self.layers.append(Layer(i, self.vector(tensors, pre + "norm1", cfg.width), mixer, norm2, mlp))
        self.runs = self.layers
        self.final_norm = self.vector(tensors, "final.norm", cfg.width)
        self.head = mo.padded_weight(self.shaped(tensors, "head", cfg.vocab, cfg.width), dtype, device)
        self.vocab_size = cfg.vocab

    def _mixer(self, spec: LayerSpec, get):
        m, cfg, rot = spec.mixer, self.config, spec.mixer["rot"]
        if spec.type == "latent_attention":
            return LatentAttention(get, cfg.width, m["heads"], m["dim"], m["vdim"], None, m["kv_rank"], m["scale"], 0, cfg.eps,
                                   self.dtype, self.device, rot_dim=m["rot_dim"], rope=self.rotary_table(rot["base"], rot["dims"]),
                                   kv_from=m["kv_from"], gate="heads", gain=cfg.gain)
        return GroupedAttention(get, cfg.width, m["heads"], m["kv_heads"], m["dim"], m["vdim"], m["scale"], m["mask"]["size"], cfg.eps,
                                self.dtype, self.device, rope=self.rotary_table(rot["base"], rot["dims"], rot["scaling"]),
                                rot_dims=rot["dims"], keep=m["mask"]["keep_first"], softcap=m["softcap"], sink=True, biased=True,
                                norm="projection", gain=cfg.gain)

    def _mlp(self, mlp: dict, get):
        cfg = self.config
        if mlp["kind"] == "dense":
            return GatedFeedForward(get, cfg.width, mlp["ff"], "silu", self.dtype, self.device, gain=cfg.gain)
        r, shared = mlp["router"], mlp["shared"]
        return RoutedExperts(get, cfg.width, mlp["expert"]["ff"], r["experts"], r["top"], r["identity"],
                             None if shared is None else shared["ff"], self.dtype, self.device, gain=cfg.gain)

    @classmethod
    def random(cls, config: dict, seed: int = 0, dtype=torch.bfloat16, device="cuda") -> "Genedra":
        """Random weights of the configuration's shapes (tests, benchmarks)."""
        return cls(config, RandomTensors(config, seed, device), dtype, device)

    # ------------------------------------------------------------------------------ serving hook
    def serving_backend(self):
        from ..serving.backends import PreNormLayers
        return PreNormLayers(self)


def RandomTensors(config: dict, seed: int = 0, device="cpu"):
    """Random weights on demand (``layered.RandomTensors``); what is stored around zero or added (norms of the layers, biases,
    corrections, sinks) is small."""
    def special(name, shape, kw):
        last = name.split(".")[-1]
        if last in ("norm1", "norm2", "b", "sink") or name == "final.norm":
            return (0.1 * torch.randn(shape, **kw)).to(torch.bfloat16)
        return (0.01 * torch.randn(shape, **kw)).to(torch.bfloat16) if last == "correction" else None
    return layered.RandomTensors(tensor_shapes(GenedraConfig.from_dict(config)), seed, device, special)


def tensor_shapes(cfg: GenedraConfig) -> dict[str, tuple[int, ...]]:
    """Name and shape of every tensor of a model of this configuration."""
    w = cfg.width
    out = {"embed": (cfg.vocab, w)}
    for i, spec in enumerate(cfg.layers):
        m, mlp, pre = spec.mixer, spec.mlp, f"l{i}."
        heads, dim, he = m["heads"], m["dim"], m["heads"] * m["vdim"]
        out[pre + "norm1"] = (w,)
        if mlp is not None:
            out[pre + "norm2"] = (w,)
        if spec.type == "latent_attention":
            kvr, rd = m["kv_rank"], m["rot_dim"]
            mix = {"q": (heads * (dim + rd), w)}
            if m["kv_from"] is None:
                mix.update({"dkv": (kvr + rd, w), "dkv.norm": (kvr,)})
            mix.update({"uk": (heads * dim, kvr), "uv": (he, kvr), "g": (heads, w), "o": (w, he)})
        else:
            kv = m["kv_heads"]
            mix = {}
            for name, rows in (("q", heads * dim), ("k", kv * dim), ("v", kv * m["vdim"])):
                mix.update({name: (rows, w), name + ".b": (rows,)})
            mix.update({"q.norm": (heads * dim,), "k.norm": (kv * dim,), "sink": (heads,), "o": (w, he), "o.b": (w,)})
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if mlp is None:
            continue
        if mlp["kind"] == "dense":
            ff = {"gate": (mlp["ff"], w), "up": (mlp["ff"], w), "down": (w, mlp["ff"])}
        else:
            f, r = mlp["expert"]["ff"], mlp["router"]
            ff = {f"e{e}.{k}": v for e in range(r["experts"]) for k, v in (("up", (f, w)), ("down", (w, f)))}
            ff.update({"router": (r["experts"] + r["identity"], w), "correction": (r["experts"] + r["identity"],)})
            if mlp["shared"] is not None:
                f = mlp["shared"]["ff"]
                ff.update({"shared.up": (f, w), "shared.down": (w, f), "shared.sg": (1, w)})
        out.update({pre + "mlp." + k: v for k, v in ff.items()})
    out["final.norm"] = (w,)
    out["head"] = (cfg.vocab, w)
    return out
