"""Small Genedra configurations and weights for the tests (nothing here comes from the package's model code); schedules, feeding and
errors are those of ``tedirax_helpers``."""
from __future__ import annotations

import torch

import genedra_oracle as O
from tedirax_helpers import alone, cut, error, feed, mixed, prompts  # noqa: F401


def latent(heads, dim, vdim, kv_rank, rot_dim, scale=None, base=500.0, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "rot_dim": rot_dim,
         "scale": (dim + rot_dim) ** -0.5 if scale is None else scale, "rot": {"base": base, "dims": rot_dim}}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mlp": mlp, "mixer": m}


def attention(heads, kv, dim, vdim, size, keep, cap, dims, factor=3.0, base=900.0, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp,
            "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": 1.5 * dim ** -0.5 if scale is None else scale,
                      "softcap": cap, "mask": {"size": size, "keep_first": keep},
                      "rot": {"base": base, "dims": dims, "scaling": {"factor": factor}}}}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(ff, experts, top, identity, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "identity": identity}, "shared": {"ff": shared}}


def config(vocab, width, layers, eps=1e-5, embed=3.0, mult=0.7, cap=20.0):
    return {"architecture": "Genedra", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "residual_mult": mult, "logit_softcap": cap, "layers": layers}


CONFIGS = {
    # every size its own, nothing a multiple of anything
    "odd": config(101, 44, [attention(6, 2, 11, 9, 5, 3, 2.5, 6, mlp=moe(13, 5, 3, 2, 7)), latent(3, 11, 7, 21, 6, mlp=dense(17)),
                            latent(5, 9, 13, 21, 6, kv_from=1, mlp=moe(9, 4, 2, 1, 15)), attention(3, 3, 10, 14, 40, 0, 30.0, 10, factor=1.0),
                            latent(2, 6, 5, 10, 2, base=60.0), latent(4, 11, 6, 21, 6, scale=0.4, kv_from=1, mlp=moe(6, 3, 3, 3, 5))],
                  eps=1e-4, embed=1.0, mult=1.0, cap=7.0),
    # sizes the tensor-core kernels take
    "tiles": config(203, 96, [latent(6, 40, 56, 72, 24, mlp=moe(40, 6, 2, 1, 24)), attention(6, 2, 48, 24, 33, 5, 8.0, 16, mlp=dense(72)),
                              latent(3, 72, 40, 72, 24, kv_from=0, mlp=moe(24, 3, 4, 2, 24)), attention(4, 1, 24, 72, 70, 1, 50.0, 8)]),
    # heads of 128 with 64 rotated dimensions more, more heads than one group of the decode kernels, windows and kept tokens of
    # several key tiles
    "wide": config(160, 128, [latent(20, 128, 128, 128, 64, mlp=moe(64, 8, 3, 2, 40)),
                              attention(18, 1, 128, 80, 150, 130, 15.0, 64, mlp=moe(32, 4, 1, 1, 64)), latent(4, 80, 128, 256, 32, mlp=dense(64)),
                              latent(17, 128, 96, 128, 64, scale=0.1, kv_from=0)], embed=10.0, mult=0.3),
    # one kind of layer each
    "attention only": config(64, 24, [attention(2, 2, 16, 16, 1, 2, 5.0, 16, mlp=dense(8)), attention(3, 1, 8, 24, 64, 200, 3.0, 4)]),
    "latent only": config(64, 32, [latent(2, 16, 16, 24, 8, mlp=moe(8, 2, 1, 1, 16)), latent(1, 8, 24, 24, 8, kv_from=0)]),
}


def tensors(cfg, seed=0, steer=False):
    """Random bf16 weights; projections, biases and sinks are scaled so that attention scores spread over several units and a sink takes
    a visible share.

    ``steer``: the routers read columns of the residual stream that hold a level per token and output, which no sublayer writes, so that
    no choice is close and 16-bit rounding cannot change it."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    mat = lambda o, i, gain=1.0: (gain * torch.randn(o, i, generator=g) * i ** -0.5).to(torch.bfloat16)
    vec = lambda n, mean=0.0, std=0.3: (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)
    out = {"embed": torch.randn(cfg["vocab"], w, generator=g).to(torch.bfloat16)}
    moes = [la["mlp"]["router"] for la in cfg["layers"] if la["mlp"] and la["mlp"]["kind"] == "moe"]
    held = max([r["experts"] + r["identity"] for r in moes], default=0) if steer else 0
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, pre = layer["mixer"], layer["mlp"], f"l{i}."
        heads, dim, he = m["heads"], m["dim"], m["heads"] * m["vdim"]
        out[pre + "norm1"] = vec(w)
        if layer["type"] == "latent_attention":
            kvr, rd = m["kv_rank"], m["rot_dim"]
            mix = {"q": mat(heads * (dim + rd), w, 1.5)}
            if m.get("kv_from") is None:
                mix.update({"dkv": mat(kvr + rd, w), "dkv.norm": vec(kvr, 1.0)})
            mix.update({"uk": mat(heads * dim, kvr, 1.5), "uv": mat(he, kvr), "g": mat(heads, w), "o": mat(w, he)})
        else:
            kv, mix = m["kv_heads"], {}
            for name, rows in (("q", heads * dim), ("k", kv * dim), ("v", kv * m["vdim"])):
                mix.update({name: mat(rows, w), name + ".b": vec(rows)})
            mix.update({"q.norm": vec(heads * dim, 1.0), "k.norm": vec(kv * dim, 1.0), "sink": vec(heads, 1.0, 1.5), "o": mat(w, he),
                        "o.b": vec(w)})
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if mlp and mlp["kind"] == "dense":
            ff = mlp["ff"]
            out.update({pre + "norm2": vec(w), pre + "mlp.gate": mat(ff, w), pre + "mlp.up": mat(ff, w), pre + "mlp.down": mat(w, ff)})
        elif mlp:
            ff, r, sh = mlp["expert"]["ff"], mlp["router"], mlp["shared"]["ff"]
            n = r["experts"] + r["identity"]
            out.update({pre + "norm2": vec(w), pre + "mlp.router": mat(n, w, 1.5), pre + "mlp.correction": vec(n, 0.0, 0.08)})
            for e in range(r["experts"]):
                out.update({f"{pre}mlp.e{e}.up": mat(ff, w, 1.5), f"{pre}mlp.e{e}.down": mat(w, ff, 1.5)})
            out.update({pre + "mlp.shared.up": mat(sh, w, 1.5), pre + "mlp.shared.down": mat(w, sh, 1.5), pre + "mlp.shared.sg": mat(1, w)})
            if held:
                order = torch.randperm(held, generator=g)[:n]
                rows = torch.zeros(n, w)
                rows[torch.arange(n), w - held + order] = 1.5
                out[pre + "mlp.router"], out[pre + "mlp.correction"] = rows.to(torch.bfloat16), vec(n, 0.0, 0.004)
    out["final.norm"], out["head"] = vec(w), mat(cfg["vocab"], w)
    if held:
        levels = torch.linspace(-1.5, 1.5, held)
        out["embed"][:, w - held:] = torch.stack([levels[torch.randperm(held, generator=g)] for _ in range(cfg["vocab"])]).to(torch.bfloat16)
        for name, t in out.items():
            if name.endswith((".norm1", ".norm2")):
                t[w - held:] = 0
            elif name.endswith((".o", ".down")) or name.endswith(".o.b"):
                t[w - held:] = 0
    return out


def closest_call(cfg, ts, seqs):
    """Smallest difference between the last chosen and the first unchosen output of any router, relative to the latter's score."""
    least, plain = [float("inf")], O.route

    def watched(h, w_router, correction, top):
        s = torch.softmax(h @ w_router.T, -1)
        if top < s.shape[1]:
            c = (s + correction).sort(-1, descending=True)
            gap = (c.values[:, top - 1] - c.values[:, top]) / s.gather(1, c.indices[:, top:top + 1])[:, 0]
            least[0] = min(least[0], float(gap.min()))
        return plain(h, w_router, correction, top)
    O.route = watched
    try:
        expected(cfg, ts, seqs)
    finally:
        O.route = plain
    return least[0]


def expected(cfg, ts, seqs):
    o = O.Oracle(cfg, ts)
    return [o.logits(s) for s in seqs]
