"""Small Beledra configurations and weights for the tests (nothing here comes from the package's model code); schedules, feeding and
errors are those of ``tedirax_helpers``."""
from __future__ import annotations

import torch

from beledra_oracle import Oracle
from tedirax_helpers import alone, cut, error, feed, mixed, prompts  # noqa: F401


def mlstm(heads, dim, vdim, cap=10.0, mlp=None):
    return {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}}


def attention(heads, kv, dim, vdim, size, bias_max, scale=None, mlp=None, rows=8):
    """``rows``: of the distance table (a tensor's shape, not a setting)."""
    return {"type": "attention", "mlp": mlp, "rows": rows,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.5 * dim ** -0.5 if scale is None else scale,
                      "mask": {"size": size}, "bias_max": bias_max}}


def yarn(factor=4.0, original=64, fast=8.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def difference(heads, kv, dim, vdim, size, dims, diff=0.3, base=500.0, scale=None, scaling=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.5 * dim ** -0.5 if scale is None else scale,
         "mask": {"size": size}, "diff": diff, "rot": {"base": base, "dims": dims, "scaling": scaling or yarn()}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention_2", "mlp": mlp, "mixer": m}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def config(vocab, width, layers, eps=1e-5):
    return {"architecture": "Beledra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers}


CONFIGS = {
    # every size its own, nothing a multiple of anything
    "odd": config(101, 44, [mlstm(3, 10, 7, 4.0, dense(13)), attention(6, 3, 11, 9, 5, 14, mlp=dense(17), rows=6),
                            difference(4, 2, 10, 7, 9, 6, mlp=dense(9)), attention(2, 2, 6, 13, 40, 20, rows=10),
                            difference(6, 2, 10, 7, 21, 6, diff=0.7, kv_from=2), mlstm(1, 5, 11)], eps=1e-4),
    # sizes the tensor-core kernels take; values and keys of different sizes; shared keys under a wider window
    "tiles": config(203, 96, [difference(6, 3, 40, 24, 33, 16, mlp=dense(72)), mlstm(2, 48, 24, 15.0),
                              attention(4, 1, 24, 72, 70, 40, mlp=dense(40), rows=16),
                              difference(3, 3, 40, 24, 150, 16, diff=0.55, kv_from=0, mlp=dense(24)), mlstm(3, 24, 56, 6.0)]),
    # heads of 128, more query vectors per key head than one group of the decode kernel
    "wide": config(160, 128, [mlstm(2, 128, 128, 15.0, dense(64)), difference(20, 1, 128, 128, 150, 64, scaling=yarn(8.0, 256, 16.0, 2.0)),
                              attention(18, 1, 128, 80, 129, 256, rows=32, mlp=dense(48)), mlstm(1, 64, 72)]),
    # one kind of layer each
    "attention only": config(64, 24, [attention(2, 2, 16, 16, 1, 30, mlp=dense(8)), attention(3, 1, 8, 24, 64, 33, rows=5)]),
    "difference only": config(64, 24, [difference(2, 2, 16, 16, 64, 16, diff=0.0, mlp=dense(8)),
                                       difference(1, 1, 24, 8, 3, 2), difference(4, 2, 16, 16, 7, 16, kv_from=0)]),
    "memory only": config(64, 32, [mlstm(1, 16, 16), mlstm(2, 8, 24, 3.0, dense(16))]),
}


def tensors(cfg, seed=0):
    """Random bf16 weights; distance tables and gates spread widely, so that a wrong bucket or a lost state shows."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    mat = lambda o, i, gain=1.0: (gain * torch.randn(o, i, generator=g) * i ** -0.5).to(torch.bfloat16)
    vec = lambda n, mean=1.0, std=0.3: (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)
    out = {"embed": torch.randn(cfg["vocab"], w, generator=g).to(torch.bfloat16)}
    for i, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{i}."
        heads, dim, he = m["heads"], m["dim"], m["heads"] * m["vdim"]
        out[pre + "norm1"] = vec(w)
        if layer["type"] == "mlstm":
            hd = heads * dim
            mix = {"q": mat(hd, w), "k": mat(hd, w), "v": mat(he, w), "g": mat(he, w), "o": mat(w, he), "norm": vec(he),
                   "i": mat(heads, w, 0.5), "i.b": vec(heads, 0.0, 1.0), "f": mat(heads, w, 0.7), "f.b": vec(heads, 3.0, 1.0)}
        else:
            maps = 1 if layer["type"] == "attention" else 2
            mix = {"q": mat(heads * maps * dim, w), "q.norm": vec(dim), "o": mat(w, he)}
            if m.get("kv_from") is None:
                mix.update({"k": mat(m["kv_heads"] * maps * dim, w), "v": mat(m["kv_heads"] * m["vdim"], w), "k.norm": vec(dim)})
            if maps == 1:
                mix["rel"] = (1.5 * torch.randn(layer["rows"], heads, generator=g)).to(torch.bfloat16)
            else:
                mix.update({k: vec(dim, 0.0, 0.2) for k in ("lq1", "lk1", "lq2", "lk2")})
                mix["g"] = mat(he, w)
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if layer["mlp"]:
            ff = layer["mlp"]["ff"]
            out.update({pre + "norm2": vec(w), pre + "mlp.gate": mat(ff, w), pre + "mlp.up": mat(ff, w), pre + "mlp.down": mat(w, ff)})
    out["final.norm"], out["head"] = vec(w), mat(cfg["vocab"], w)
    return out


def settings(cfg):
    """The configuration as a user writes it: the rows of a distance table are no setting."""
    return {**cfg, "layers": [{k: v for k, v in layer.items() if k != "rows"} for layer in cfg["layers"]]}


def expected(cfg, ts, seqs):
    o = Oracle(cfg, ts)
    return [o.logits(s) for s in seqs]
