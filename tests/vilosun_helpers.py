"""Small Vilosun configurations and weights for the tests (nothing here comes from the package's model code); schedules, feeding and
errors are those of ``tedirax_helpers``."""
from __future__ import annotations

import torch

import tedirax_helpers
import vilosun_oracle as O
from tedirax_helpers import alone, cut, error, mixed, prompts  # noqa: F401


def attention(heads, kv, dim, vdim, size, conv, v_mix=True, scale=None, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv, "v_mix": v_mix,
                                                       "scale": 1.5 * dim ** -0.5 if scale is None else scale, "mask": {"size": size}}}


def delta(heads, kv, dim, vdim, conv, mlp=None):
    return {"type": "delta", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "conv": conv}}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, groups, layers, eps=1e-5, embed=3.0, buckets=37, mul=(5, 3), logit=0.5):
    return {"architecture": "Vilosun", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups}, "logit_scale": logit,
            "embedding": {"scale": embed, "bigram": {"buckets": buckets, "mul_prev": mul[0], "mul_cur": mul[1]}}, "layers": layers}


CONFIGS = {
    # every size its own, nothing a multiple of anything; the first layer that mixes values is not the first attention
    "odd": config(101, 45, 5, [attention(6, 2, 11, 9, 5, 2, False, mlp=moe(13, 5, 3)), delta(6, 3, 10, 7, 5), attention(4, 2, 10, 13, 40, 3, scale=-0.4),
                               delta(2, 1, 13, 12, 3, mlp=moe(9, 4, 4)), attention(6, 2, 7, 13, 3, 6, mlp=moe(6, 3, 1)), delta(3, 3, 5, 11, 1)],
                  eps=1e-4, embed=1.0, mul=(40000001, 7), logit=1.0),
    # sizes the tensor-core kernels take
    "tiles": config(203, 96, 3, [delta(6, 3, 40, 56, 4, mlp=moe(40, 6, 2)), attention(6, 2, 48, 24, 33, 3, mlp=moe(24, 3, 3)),
                                 delta(4, 4, 64, 64, 2), attention(4, 2, 24, 24, 70, 4, mlp=moe(72, 5, 1)), delta(2, 1, 104, 24, 6)], buckets=500, mul=(203, 1)),
    # heads of 128, more query heads than one group of the decode kernels, chunks of several key tiles
    "wide": config(160, 128, 1, [delta(4, 2, 128, 128, 4, mlp=moe(64, 8, 3)), attention(34, 2, 128, 80, 150, 3, mlp=moe(32, 4, 1)),
                                 delta(2, 2, 104, 128, 1), attention(4, 2, 72, 80, 64, 1), attention(2, 2, 128, 80, 1000, 4, scale=0.1)], logit=0.1),
    # one kind of layer each
    "attention only": config(64, 24, 4, [attention(2, 2, 16, 16, 1, 1, mlp=moe(8, 2, 1)), attention(3, 1, 8, 24, 200, 2, False)], buckets=1),
    "delta only": config(64, 32, 2, [delta(2, 2, 16, 16, 4, mlp=moe(8, 2, 1)), delta(1, 1, 8, 24, 4)]),
}


def tensors(cfg, seed=0, steer=False):
    """Random bf16 weights; projections, slopes' rivals (queries and keys) and gates are scaled so that scores spread over several units,
    decays last from two to some hundred tokens.

    ``steer``: the routers read columns of the residual stream that hold a level per token and expert, which no sublayer writes, so that
    no choice is close and 16-bit rounding cannot change it."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    mat = lambda o, i, gain=1.0: (gain * torch.randn(o, i, generator=g) * i ** -0.5).to(torch.bfloat16)
    vec = lambda n, mean=0.0, std=0.3: (mean + std * torch.randn(n, generator=g)).to(torch.bfloat16)

    def filt(n, taps):
        t = 0.4 * torch.randn(n, taps, generator=g)
        t[:, -1] += 1.0
        return t.to(torch.bfloat16)
    out = {"embed": torch.randn(cfg["vocab"], w, generator=g).to(torch.bfloat16),
           "bigram": torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, w, generator=g).to(torch.bfloat16)}
    moes = [la["mlp"]["router"] for la in cfg["layers"] if la["mlp"]]
    held = max([r["experts"] for r in moes], default=0) if steer else 0
    for i, layer in enumerate(cfg["layers"]):
        m, mlp, pre = layer["mixer"], layer["mlp"], f"l{i}."
        heads, kv, dim, he = m["heads"], m["kv_heads"], m["dim"], m["heads"] * m["vdim"]
        sub = lambda n: {f"norm{n}": vec(w, 1.0), f"norm{n}b": vec(w, 0.8), f"rg{n}": mat(w, w), f"rg{n}.b": vec(w)}
        mix = {}
        if layer["type"] == "attention":
            rows = (("q", heads * dim, 1.5), ("k", kv * dim, 1.5), ("v", kv * m["vdim"], 1.0))
            for name, n, _ in rows:
                mix[name + ".b"] = vec(n)
            mix.update({"temp": vec(heads, 1.0), "g": mat(heads, w), "o": mat(w, he)})
            if m["v_mix"]:
                mix["vmix"] = torch.tensor(0.35 + 0.1 * i).to(torch.bfloat16)
        else:
            rows = (("q", kv * dim, 1.5), ("k", kv * dim, 1.5), ("v", he, 1.0))
            mix.update({"a": mat(heads, w), "b": mat(heads, w, 1.5), "A_log": vec(heads, -1.0, 1.0), "dt_bias": vec(heads, -2.0, 1.0),
                        "norm": vec(m["vdim"], 1.0), "g": mat(he, w), "o": mat(w, he)})
        for name, n, gain in rows:
            mix.update({name: mat(n, w, gain), name + ".conv": filt(n, m["conv"])})
        out.update({pre + k: v for k, v in sub(1).items()})
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if not mlp:
            continue
        out.update({pre + k: v for k, v in sub(2).items()})
        ff, n = mlp["expert"]["ff"], mlp["router"]["experts"]
        out.update({pre + "mlp.router": mat(n, w, 1.5), pre + "mlp.router.b": vec(n, 0.0, 0.5)})
        for e in range(n):
            out.update({f"{pre}mlp.e{e}.gate": mat(ff, w, 1.5), f"{pre}mlp.e{e}.up": mat(ff, w, 1.5), f"{pre}mlp.e{e}.down": mat(w, ff, 1.5)})
        if held:
            order = torch.randperm(held, generator=g)[:n]
            rows = torch.zeros(n, w)
            rows[torch.arange(n), w - held + order] = 2.0
            out[pre + "mlp.router"], out[pre + "mlp.router.b"] = rows.to(torch.bfloat16), vec(n, 0.0, 0.01)
    out["final.norm"], out["head"] = vec(w, 1.0), mat(cfg["vocab"], w)
    if held:
        levels = torch.linspace(-2.0, 2.0, held)
        out["embed"][:, w - held:] = torch.stack([levels[torch.randperm(held, generator=g)] for _ in range(cfg["vocab"])]).to(torch.bfloat16)
        out["bigram"][:, w - held:] = 0
        for name, t in out.items():
            if name.endswith(("norm1b", "norm2b")):
                t[w - held:] = 0
            elif name.endswith(".norm2"):
                t[w - held:] = 1
    return out


def closest_call(cfg, ts, seqs):
    """Smallest difference between the last chosen and the first unchosen logit of any router."""
    least, plain = [float("inf")], O.route

    def watched(z, top):
        if top < z.shape[1]:
            c = z.sort(-1, descending=True).values
            least[0] = min(least[0], float((c[:, top - 1] - c[:, top]).min()))
        return plain(z, top)
    O.route = watched
    try:
        expected(cfg, ts, seqs)
    finally:
        O.route = plain
    return least[0]


def expected(cfg, ts, seqs):
    o = O.Oracle(cfg, ts)
    return [o.logits(s) for s in seqs]


def poison(entries):
    """Nothing may be read that was not written by its own request."""
    for e in entries:
        if isinstance(e, tuple):
            poison(e)
        elif e.dtype == torch.int32:
            e.fill_(10 ** 6 + 7)
        else:
            e.fill_(float("nan"))


def feed(engine, seqs, schedule, spoil=True):
    if spoil:
        poison(engine.cache.entries)
    return tedirax_helpers.feed(engine, seqs, schedule)
