"""Small Tedirax configurations, weights and schedules for the tests (nothing here comes from the package's model code)."""
from __future__ import annotations

import numpy as np
import torch

from tedirax_oracle import Oracle


def retention(heads, dim, vdim, decay, base=1000.0, dims=None, mlp=None):
    return {"type": "retention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay,
                                                       "rot": {"base": base, "dims": dim if dims is None else dims}}}


def latent(heads, dim, vdim, q_rank, kv_rank, size, scale=None, mlp=None):
    return {"type": "latent_attention", "mlp": mlp,
            "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
                      "scale": dim ** -0.5 if scale is None else scale, "mask": {"size": size}}}


def moe(ff, experts, top):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def config(vocab, width, layers, loop=None, eps=1e-5):
    return {"architecture": "Tedirax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "loop": loop, "layers": layers}


CONFIGS = {
    # every size its own, nothing a multiple of anything
    "odd": config(101, 44, [retention(3, 10, 7, [0.9, 0.5, 0.99], dims=6, mlp=moe(13, 5, 3)),
                            latent(5, 11, 6, 19, 21, 5, scale=0.41, mlp=moe(9, 4, 1)),
                            retention(2, 6, 9, [0.97, 0.8], base=50.0)], {"start": 1, "stop": 3, "times": 2}, eps=1e-4),
    # sizes the tensor-core kernels take, partial rotation, vdim and dim different, a loop over everything
    "tiles": config(203, 96, [latent(6, 48, 40, 56, 72, 33, mlp=moe(24, 6, 2)),
                              retention(3, 48, 24, [0.97, 0.99, 0.9], dims=16, mlp=moe(40, 3, 3))],
                    {"start": 0, "stop": 2, "times": 2}),
    # heads of 128, more heads than one group of the decode kernel, a window of several key tiles, no loop
    "wide": config(160, 128, [retention(2, 128, 128, [0.995, 0.96], dims=64, mlp=moe(64, 8, 2)),
                              latent(20, 80, 128, 64, 136, 150),
                              retention(1, 64, 72, [0.9375], mlp=moe(16, 4, 4))]),
    # one layer kind only, a window of one token, experts never chosen twice
    "latent only": config(64, 24, [latent(2, 8, 8, 16, 16, 1, mlp=moe(8, 2, 1)), latent(1, 16, 8, 8, 24, 64)]),
    "retention only": config(64, 32, [retention(1, 16, 16, [0.999])], {"start": 0, "stop": 1, "times": 3}),
}


def tensors(cfg, seed=0):
    """Random bf16 weights; projections are scaled so that attention scores spread over several units."""
    g = torch.Generator().manual_seed(seed)
    w = cfg["width"]
    mat = lambda o, i, gain=1.0: (gain * torch.randn(o, i, generator=g) * i ** -0.5).to(torch.bfloat16)
    vec = lambda n: (1 + 0.3 * torch.randn(n, generator=g)).to(torch.bfloat16)
    out = {"embed": torch.randn(cfg["vocab"], w, generator=g).to(torch.bfloat16)}
    for i, layer in enumerate(cfg["layers"]):
        m, pre = layer["mixer"], f"l{i}."
        hd, he = m["heads"] * m["dim"], m["heads"] * m["vdim"]
        out[pre + "norm1"] = vec(w)
        if layer["type"] == "retention":
            mix = {"q": mat(hd, w), "k": mat(hd, w), "v": mat(he, w), "g": mat(he, w), "o": mat(w, he)}
        else:
            qr, kr = m["q_rank"], m["kv_rank"]
            mix = {"dq": mat(qr, w), "dq.norm": vec(qr), "uq": mat(hd, qr, 1.5), "dkv": mat(kr, w), "dkv.norm": vec(kr),
                   "uk": mat(hd, kr, 1.5), "uv": mat(he, kr), "g": mat(he, w), "o": mat(w, he)}
        out.update({pre + "mix." + k: v for k, v in mix.items()})
        if layer["mlp"]:
            ff, n, top = layer["mlp"]["expert"]["ff"], layer["mlp"]["router"]["experts"], layer["mlp"]["router"]["top"]
            for e in range(n):
                out.update({f"{pre}mlp.e{e}.gate": mat(ff, w), f"{pre}mlp.e{e}.up": mat(ff, w), f"{pre}mlp.e{e}.down": mat(w, ff)})
            out[pre + "mlp.table"] = torch.stack([torch.randperm(n, generator=g)[:top] for _ in range(cfg["vocab"])]).to(torch.int32)
    out["final.norm"], out["head"] = vec(w), mat(cfg["vocab"], w)
    return out


def prompts(cfg, lengths, seed=1):
    g = torch.Generator().manual_seed(seed)
    return [torch.randint(0, cfg["vocab"], (n,), generator=g).tolist() for n in lengths]


def error(got, want):
    """Worst row: root mean square of the difference (mean taken off) over that of the expected logits."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    w = want - want.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / w.pow(2).mean(-1).sqrt()
    return float("inf") if torch.isnan(e).any() else float(e.max())


def expected(cfg, ts, seqs):
    o = Oracle(cfg, ts)
    return [o.logits(s) for s in seqs]


def feed(engine, seqs, schedule, poison=False):
    """Run ``schedule`` (a list of steps, each a list of (sequence, tokens)) through ``engine.extend``, all logits wanted;
    a sequence is closed when its tokens are used up.  Returns the logits per sequence."""
    if poison:
        # nothing may be read that was not written by its own request (the zero padding of a latent is not data)
        for run, e in zip(engine.backend.model.runs, engine.cache.entries):
            pad = hasattr(run.mixer, "kv_rank") and not run.mixer.rot
            e[..., :run.mixer.kv_rank if pad else e.shape[-1]] = float("nan")
    at, live, got = [0] * len(seqs), {}, [[] for _ in seqs]
    for step in schedule:
        entries = []
        for i, n in step:
            if i not in live:
                live[i] = engine.open(i)
            entries.append((live[i], seqs[i][at[i]:at[i] + n], list(range(n))))
        logits = engine.extend(entries)
        row = 0
        for i, n in step:
            got[i].append(logits[row:row + n].float().cpu())
            row += n
            at[i] += n
            if at[i] == len(seqs[i]):
                engine.close(live.pop(i))
    assert all(a == len(s) for a, s in zip(at, seqs))
    return [torch.cat(g) for g in got]


def cut(length, sizes):
    """Portion sizes that go round ``sizes`` until ``length`` is used up."""
    out, k = [], 0
    while sum(out) < length:
        out.append(min(sizes[k % len(sizes)], length - sum(out)))
        k += 1
    return out


def alone(i, length, sizes):
    return [[(i, n)] for n in cut(length, sizes)]


def mixed(lengths, sizes, live=3, seed=0):
    """Up to ``live`` requests at a time, each cut by its own sizes; a request now and then sits a step out."""
    rng = np.random.default_rng(seed)
    parts = [cut(n, sizes[i % len(sizes)]) for i, n in enumerate(lengths)]
    waiting, active, steps = list(range(len(lengths))), [], []
    while waiting or active:
        while waiting and len(active) < live:
            active.append(waiting.pop(0))
        run = [i for i in active if rng.random() < 0.8] or active[:1]
        steps.append([(i, parts[i].pop(0)) for i in run])
        active = [i for i in active if parts[i]]
    return steps
