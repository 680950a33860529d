"""Genedra at the sizes of ``bench_layers``: its configuration, and its kernels beside the like kernels of the other models, each
against its roofline (measured as ``bench_layers`` describes)."""
from __future__ import annotations

import torch

from . import mixer_ops as mo
from . import native
from .bench_layers import (CONTEXT, DECODE_BATCHES, EXPERTS, PROMPT_LEN, PROMPTS, SIZES, TOP, _bf, _expert_kernels, _residual_kernel,
                           _Table, graph_ms, peaks)
from .bench_ops import timeit

GROUP = 4                        # query heads per key/value head
ROT, KEEP, CAP, IDENTITY = 64, 4, 50.0, 1


def genedra_config(s: dict) -> dict:
    """Three layers over and over: latent attention, latent attention on the cache of the one before, windowed attention.  The first
    layer is dense with the TransformerLM's width; in the others the two chosen experts (two matrices each) and the shared one have
    as many active weights."""
    heads, f = s["heads"], s["ff"] // TOP
    lat = {"heads": heads, "dim": 128, "vdim": 128, "kv_rank": s["kv_rank"], "rot_dim": ROT, "scale": (128 + ROT) ** -0.5,
           "rot": {"base": 10000.0, "dims": ROT}}
    att = {"heads": heads, "kv_heads": heads // GROUP, "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": CAP,
           "mask": {"size": s["window"], "keep_first": KEEP}, "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0}}}
    moe = {"kind": "moe", "expert": {"ff": f}, "router": {"experts": EXPERTS, "top": TOP, "identity": IDENTITY}, "shared": {"ff": f}}
    layers = []
    for i in range(s["runs"]):
        mlp = {"kind": "dense", "ff": s["ff"]} if i == 0 else moe
        if i % 3 == 2:
            layers.append({"type": "attention", "mlp": mlp, "mixer": att})
        else:
            layers.append({"type": "latent_attention", "mlp": mlp, "mixer": {**lat, "kv_from": i - 1} if i % 3 == 1 else lat})
    return {"architecture": "Genedra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "embedding": {"scale": 8.0},
            "residual_mult": 0.25, "logit_softcap": 30.0, "layers": layers}


def _grouped(s):
    """Beledra's attention with a distance bias, and Genedra's."""
    heads, kv, win = s["heads"], s["heads"] // GROUP, s["window"]
    bias = torch.randn(heads, min(win, 1024), device="cuda")
    return (mo.AttentionShape(heads, kv, 1, 128, 128, 64, 128 ** -0.5, win, 1e-6, bias=bias),
            mo.AttentionShape(heads, kv, 1, 128, 128, 64, 128 ** -0.5, win, 1e-6, keep=KEEP, softcap=CAP,
                              sink=torch.randn(heads, device="cuda"), whole_norm=True))


def kernels(size: str) -> dict:
    s, pk = SIZES[size], peaks()
    t = _Table(pk)
    with torch.no_grad():
        _prompt_kernels(s, t)
        torch.cuda.empty_cache()
        for b in DECODE_BATCHES:
            _decode_kernels(s, t, b)
            torch.cuda.empty_cache()
    native.check_status()
    return {"size": size, "peaks": pk, "kernels": t.rows}


def _prompt_kernels(s, t):
    w, heads, rows, ff = s["width"], s["heads"], PROMPTS * PROMPT_LEN, s["ff"]
    hd, win, kvr, f = heads * 128, s["window"], s["kv_rank"], s["ff"] // TOP
    cu = torch.arange(PROMPTS + 1, dtype=torch.int32, device="cuda") * PROMPT_LEN
    pos = torch.arange(PROMPT_LEN, dtype=torch.int32, device="cuda").repeat(PROMPTS)
    slots = torch.arange(rows, device="cuda")
    tables = torch.arange(rows // 64, device="cuda").int().view(PROMPTS, PROMPT_LEN // 64)
    seen, pairs = PROMPTS * (win * (win + 1) / 2 + (PROMPT_LEN - win) * win), PROMPTS * PROMPT_LEN * (PROMPT_LEN + 1) / 2
    kept = seen + PROMPTS * max(0, PROMPT_LEN - win - KEEP) * KEEP
    # attention over keys
    q, kv, gate, o = _bf(rows, hd), _bf(rows, 2 * hd), _bf(rows, hd), _bf(rows, hd)
    t.add(f"flash_window_fwd, window {win}, gate (Tedirax)", "-",
          timeit(lambda: mo.window_attention(q, kv, cu, cu, PROMPT_LEN, heads, 128, 128, win, 128 ** -0.5, o, gate)), rows * hd * 10, 4 * seen * hd)
    qr, kr, hg = _bf(rows, heads * (128 + ROT)), _bf(rows, kvr + ROT), _bf(rows, heads)
    t.add("flash_window_fwd, causal, rotated part, gate per head", "flash_window_fwd",
          timeit(lambda: mo.window_attention(qr, kv, cu, cu, PROMPT_LEN, heads, 128, 128, 0, (128 + ROT) ** -0.5, o, hg, None,
                                             (kr, ROT, hd, ROT, kvr))), rows * (hd * 8 + heads * ROT * 2 + ROT * 2), 2 * pairs * heads * (256 + ROT))
    del q, kv, qr, kr
    for name, like, a in zip(("distance bias (Beledra)", "kept tokens, cap, sink"), ("-", "grouped_prefill, distance bias"), _grouped(s)):
        q, cache = _bf(rows, heads * a.q_pitch), _bf(rows // 64, 64, a.cache_width)
        t.add(f"grouped_prefill, window {win}, {name}", like,
              timeit(lambda: mo.attention_portions(q, a, cache, pos, cu, PROMPT_LEN, tables, o)), rows * (q.shape[1] + a.cache_width + hd) * 2,
              4 * (kept if a.keep else seen) * hd)
    del q, cache, gate, o
    # experts
    a, wgu = _bf(rows, w), _bf(2 * ff, w)
    t.add("gate|up GEMM (TransformerLM)", "-", timeit(lambda: native.gemm(a, wgu, "nt")), (rows * w + 2 * ff * w + rows * 2 * ff) * 2, 4.0 * rows * w * ff)
    h, wd = _bf(rows, ff), _bf(w, ff)
    res = torch.zeros(rows, w, device="cuda")
    t.add("down GEMM into the fp32 residual", "-", timeit(lambda: mo.linear(h, wd, out=res, accumulate=True)),
          (rows * ff + ff * w) * 2 + rows * w * 8, 2.0 * rows * w * ff)
    t.add("down GEMM into the fp32 residual, gain", "down GEMM", timeit(lambda: mo.linear(h, wd, out=res, accumulate=True, alpha=0.25)),
          (rows * ff + ff * w) * 2 + rows * w * 8, 2.0 * rows * w * ff)
    del wgu, h, wd, res
    _expert_kernels(s, t, rows, torch.randint(0, s["vocab"], (rows,), device="cuda"))
    n, outputs = rows * TOP, EXPERTS + IDENTITY
    wr, corr = _bf(outputs + 1, w), torch.zeros(outputs, device="cuda")
    t.add("router GEMM (fp32 out)", "-", timeit(lambda: mo.linear(a, wr, out_dtype=torch.float32)), (rows * w + wr.numel()) * 2 + rows * outputs * 4,
          2.0 * rows * w * outputs)
    z, live, zero = torch.randn(rows, outputs, device="cuda"), torch.zeros(rows, dtype=torch.int64, device="cuda"), lambda: torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
    count = zero()
    choice, rank, weight = mo.moe_route(z, corr, live, EXPERTS, TOP, count)
    t.add("moe_route", "moe_plan", timeit(lambda: mo.moe_route(z, corr, live, EXPERTS, TOP, zero())), rows * (outputs * 4 + TOP * 12))
    t.add("moe_dispatch", "residual_norm", timeit(lambda: mo.moe_dispatch(a, choice, rank, count)), rows * w * 2 + int(count.sum()) * w * 2)
    xg, mpos, group = mo.moe_dispatch(a, choice, rank, count)
    n = int(count.sum())
    wu, wdn, su, sd = _bf(EXPERTS * f, w), _bf(EXPERTS * w, f), _bf(f, w), _bf(w, f)
    hid, sh = mo.gemm_rows(xg, wu, group, f, False, "gelu"), mo.linear(a, su, act="gelu")
    t.add("experts up + GELU", "experts gate|up", timeit(lambda: mo.gemm_rows(xg, wu, group, f, False, "gelu")), (n * w + EXPERTS * f * w + n * f) * 2, 2.0 * n * w * f)
    t.add("experts down, routed", "experts down", timeit(lambda: mo.gemm_rows(hid, wdn, group, w, False)), (n * f + EXPERTS * f * w + n * w) * 2, 2.0 * n * w * f)
    t.add("shared up + GELU", "gate|up GEMM", timeit(lambda: mo.linear(a, su, act="gelu")), (rows * w + f * w + rows * f) * 2, 2.0 * rows * w * f)
    t.add("shared down", "down GEMM", timeit(lambda: mo.linear(sh, sd)), (rows * f + f * w + rows * w) * 2, 2.0 * rows * w * f)
    del wu, wdn, hid, sh, xg
    # rows
    nw = torch.ones(w, device="cuda").bfloat16()
    t.add("rmsnorm_fwd (TransformerLM)", "-", timeit(lambda: native.rmsnorm_fwd(a, nw, 1e-6)), rows * w * 4)
    _residual_kernel(s, t, rows)
    x, y, sh = torch.randn(rows, w, device="cuda"), _bf(mo.plan_tiles(rows, EXPERTS, TOP) * mo.TILE, w), _bf(rows, w)
    ex = mo.ExpertOutputs(y, mpos, 0.0, weight, a, sh, z[:, 0])
    t.add("residual_norm with routed experts", "residual_norm", timeit(lambda: mo.residual_norm(x, nw, 1e-6, pending=ex, w_offset=1.0)),
          rows * w * (8 + 2 * TOP + 2 + 2))
    t.add("residual_norm, norm only", "rmsnorm_fwd", timeit(lambda: mo.residual_norm(x, nw, 1e-6, w_offset=1.0)), rows * w * 6)
    del y, sh, ex
    pr, nq, nkv = _bf(rows, s["q_rank"] + kvr + hd), _bf(s["q_rank"]), _bf(kvr)
    cache = torch.zeros(rows // 64, 64, kvr, dtype=torch.bfloat16, device="cuda")
    t.add("latent_norm_append (Tedirax)", "-", timeit(lambda: mo.latent_norm_append(pr, nq, nkv, 1e-6, cache, slots)), rows * (s["q_rank"] + kvr) * 4)
    pr, cache = _bf(rows, heads * (128 + ROT) + kvr + ROT + heads), torch.zeros(rows // 64, 64, kvr + ROT, dtype=torch.bfloat16, device="cuda")
    cs, qc = torch.randn(2, PROMPT_LEN, ROT // 2, device="cuda"), heads * (128 + ROT)
    t.add("latent_rotate", "latent_norm_append",
          timeit(lambda: mo.latent_rotate(pr, hd, ROT, pr, qc, qc + kvr, nkv, None, cache, cs, pos, slots, heads, kvr, kvr, ROT, 1e-6)),
          rows * (heads * ROT + kvr + ROT) * 4)
    first = torch.zeros(PROMPTS, dtype=torch.int32, device="cuda")

    def gather():
        c = torch.zeros(rows // 64, 64, kvr + ROT, dtype=torch.bfloat16, device="cuda")
        return lambda: mo.latent_gather(c, cu, first, tables, rows)
    t.add("latent_gather", "latent_gather", graph_ms(gather, rows * (kvr + ROT) * 4), rows * (kvr + ROT) * 4)
    for name, like, g in zip(("rotation (Beledra)", "whole norm, rotation"), ("-", "grouped_prep, rotation"), _grouped(s)):
        m = (g.heads + 2 * g.kv_heads) * 128
        pr, cache, cs = _bf(rows, m), torch.zeros(rows // 64, 64, g.cache_width, dtype=torch.bfloat16, device="cuda"), torch.randn(2, PROMPT_LEN, 32, device="cuda")
        wq, wk = (torch.ones(128 * (k if g.whole_norm else 1), device="cuda").bfloat16() for k in (g.heads, g.kv_heads))
        t.add(f"grouped_prep, {name}", like, timeit(lambda: mo.attention_prepare(pr, g, wq, wk, cs, pos, slots, cache)), rows * m * 4)


def _decode_kernels(s, t, b):
    w, heads, ff = s["width"], s["heads"], s["ff"]
    hd, win, kvr, f = heads * 128, min(s["window"], CONTEXT), s["kv_rank"], ff // TOP
    ctx = torch.full((b,), CONTEXT, dtype=torch.int32, device="cuda")
    pos, slots = ctx - 1, torch.zeros(b, dtype=torch.int64, device="cuda")

    def add(name, like, nbytes, flops, make):
        t.add(f"{name}, batch {b}", like, graph_ms(make, nbytes), nbytes, flops)
        torch.cuda.empty_cache()

    def tables():
        n = -(-(CONTEXT + 16) // 64)
        tb = torch.zeros(b, 32, dtype=torch.int32, device="cuda")
        tb[:, :n] = torch.randperm(b * n, device="cuda").int().view(b, n)
        return tb, b * n

    def latent(rot, window):
        def make():
            tb, pages = tables()
            ql, cache = _bf(b, heads * (kvr + rot)), _bf(pages, 64, kvr + rot)
            return lambda: mo.latent_decode(ql, cache, pos, slots, tb, heads, window, 0.1, vwidth=kvr)
        return make
    add(f"latent_decode, window {win} (Tedirax)", "-", b * (win * kvr * 2 + heads * kvr * 4), 4.0 * b * heads * win * kvr, latent(0, s["window"]))
    add(f"latent_decode, rotated part, context {CONTEXT}", "latent_decode", b * (CONTEXT * (kvr + ROT) * 2 + heads * (2 * kvr + ROT) * 2),
        2.0 * b * heads * CONTEXT * (2 * kvr + ROT), latent(ROT, 0))
    for name, like, a in zip(("distance bias (Beledra)", "kept tokens, cap, sink"), ("-", "grouped_decode, distance bias"), _grouped(s)):
        def grouped():
            tb, pages = tables()
            q, cache, o = _bf(b, heads * a.q_pitch), _bf(pages, 64, a.cache_width), _bf(b, hd)
            return lambda: mo.attention_decode(q, a, cache, pos, slots, tb, o)
        add(f"grouped_decode, window {win}, {name}", like, b * ((win + a.keep) * a.cache_width + heads * a.q_pitch + hd) * 2, 0, grouped)

    def plain(n, k, **kw):
        def make():
            x, wt = _bf(b, k), _bf(n, k)
            return lambda: mo.linear(x, wt, **kw)
        return make
    size = lambda n, k, out=2: (n * k + b * k) * 2 + b * n * out
    kvd, outputs = heads // GROUP * 128, EXPERTS + IDENTITY
    bias = torch.randn(hd + 2 * kvd, device="cuda")
    for name, like, n, k, kw in (("qkv GEMM (TransformerLM)", "-", 3 * hd, w, {}), ("gate|up GEMM (TransformerLM)", "-", 2 * ff, w, {}),
                                 ("down GEMM", "-", w, ff, {}), ("latent q|dkv|g GEMM", "qkv GEMM", heads * (128 + ROT) + kvr + ROT + heads, w, {}),
                                 ("attention q|k|v GEMM, bias", "qkv GEMM", hd + 2 * kvd, w, {"bias": bias}),
                                 ):
        add(name, like, size(n, k), 0, plain(n, k, **kw))

    def out_gemm(alpha):
        def make():
            y, wt, x = _bf(b, hd), _bf(w, hd), torch.zeros(b, w, device="cuda")
            return lambda: mo.linear(y, wt, out=x, accumulate=True, alpha=alpha)
        return make
    add("output GEMM into the fp32 residual", "-", (w * hd + b * hd) * 2 + b * w * 8, 0, out_gemm(1.0))
    add("output GEMM into the fp32 residual, gain", "output GEMM", (w * hd + b * hd) * 2 + b * w * 8, 0, out_gemm(0.25))

    def from_latent(by_head):
        def make():
            ol, wv, gate = _bf(b, heads * kvr), _bf(hd, kvr), _bf(b, heads if by_head else hd)
            return lambda: mo.gemm_heads(ol, wv, heads, kvr, 128, gate=gate)
        return make
    add("latent outputs to heads, gate (Tedirax)", "-", (heads * kvr * 128 + 2 * b * hd + b * heads * kvr) * 2, 0, from_latent(False))
    add("latent outputs to heads, gate per head", "latent outputs to heads", (heads * kvr * 128 + b * hd + b * heads * kvr) * 2, 0, from_latent(True))
    # experts
    tab = torch.rand(s["vocab"], EXPERTS, device="cuda").argsort(1)[:, :TOP].int().contiguous()
    tokens = torch.randint(0, s["vocab"], (b,), device="cuda")
    (ppos,), (pgroup,) = mo.moe_plan(tokens, slots, [tab], [EXPERTS])
    p, n = mo.plan_tiles(b, EXPERTS, TOP) * mo.TILE, b * TOP
    add("moe_plan, 1 layer (Tedirax)", "-", n * 8, 0, lambda: (lambda: mo.moe_plan(tokens, slots, [tab], [EXPERTS])))

    def route():
        h, wr, corr, counts = _bf(b, w), _bf(outputs + 1, w), torch.zeros(outputs, device="cuda"), torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
        return lambda: mo.moe_route_rows(h, wr, corr, slots, EXPERTS, TOP, counts, 1)
    add("moe_route_rows (product, choice)", "moe_plan", ((b + outputs + 1) * w + b * (outputs + 1) * 2 + b * TOP * 6) * 2, 0, route)
    z, count = torch.randn(b, outputs + 1, device="cuda"), torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
    choice, rank, weight = mo.moe_route(z, torch.zeros(outputs, device="cuda"), slots, EXPERTS, TOP, count, 1)
    m, all_experts = int(count.sum()) + b, EXPERTS + 1          # the shared expert has the others' size and joins them
    p = max(p, mo.plan_tiles(b, EXPERTS, TOP, 1) * mo.TILE)

    def dispatch():
        h = _bf(b, w)
        return lambda: mo.moe_dispatch(h, choice, rank, count, 1)
    add("moe_dispatch", "moe_plan", (b + m) * w * 2, 0, dispatch)
    _, mpos, group = mo.moe_dispatch(_bf(b, w), choice, rank, count, 1)

    def rows_gemm(rows, k, width, groups, glu, act=None):
        def make():
            xg, wt = _bf(groups.numel() * mo.TILE, k), _bf(all_experts * width * (2 if glu else 1), k)
            return lambda: mo.gemm_rows(xg, wt, groups, width, glu, act)
        return make
    add("experts gate|up + SwiGLU (Tedirax)", "-", (n * w + EXPERTS * 2 * f * w + n * f) * 2, 4.0 * n * w * f, rows_gemm(n, w, f, pgroup, True))
    add("experts up + GELU, routed and shared", "experts gate|up", (m * w + all_experts * f * w + m * f) * 2, 2.0 * m * w * f, rows_gemm(m, w, f, group, False, "gelu"))
    add("experts down (Tedirax)", "-", (n * f + EXPERTS * f * w + n * w) * 2, 2.0 * n * w * f, rows_gemm(n, f, w, pgroup, False))
    add("experts down, routed and shared", "experts down", (m * f + all_experts * f * w + m * w) * 2, 2.0 * m * w * f, rows_gemm(m, f, w, group, False))
    # rows
    nw = torch.ones(w, device="cuda").bfloat16()

    def resid(routed):
        def make():
            x, y = torch.randn(b, w, device="cuda"), _bf(p, w)
            if not routed:
                return lambda: mo.residual_norm(x, nw, 1e-6, pending=(y, ppos, 0.0), scatter=(ppos, p))
            ex = mo.ExpertOutputs(y, mpos, 0.0, weight, _bf(b, w))
            return lambda: mo.residual_norm(x, nw, 1e-6, pending=ex, w_offset=1.0)
        return make
    add("residual_norm with experts (Tedirax)", "-", b * w * (8 + 2 * TOP + 2 + 2 * TOP), 0, resid(False))
    add("residual_norm with routed experts", "residual_norm", b * w * (8 + 2 * TOP + 2 + 2), 0, resid(True))
    nq, nkv = _bf(s["q_rank"]), _bf(kvr)
    at = torch.arange(b, device="cuda") * 16

    def append():
        pr, cache = _bf(b, s["q_rank"] + kvr + hd), _bf(b, 16, kvr)
        return lambda: mo.latent_norm_append(pr, nq, nkv, 1e-6, cache, at)
    add("latent_norm_append (Tedirax)", "-", b * (s["q_rank"] + kvr) * 4, 0, append)
    cs, qc = torch.randn(2, 2048, ROT // 2, device="cuda"), heads * (128 + ROT)

    def rotate():
        pr, cache, ql = _bf(b, qc + kvr + ROT + heads), _bf(b, 16, kvr + ROT), _bf(b, heads * (kvr + ROT))
        return lambda: mo.latent_rotate(pr, hd, ROT, pr, qc, qc + kvr, nkv, ql, cache, cs, pos, at, heads, kvr, kvr, ROT, 1e-6)
    add("latent_rotate", "latent_norm_append", b * (heads * ROT + kvr + ROT) * 4, 0, rotate)
    for name, like, g in zip(("rotation (Beledra)", "whole norm, rotation"), ("-", "grouped_prep, rotation"), _grouped(s)):
        wq, wk = (torch.ones(128 * (k if g.whole_norm else 1), device="cuda").bfloat16() for k in (g.heads, g.kv_heads))

        def prep():
            pr, cache = _bf(b, hd + 2 * kvd), _bf(b, 16, g.cache_width)
            return lambda: mo.attention_prepare(pr, g, wq, wk, cs, pos, at, cache)
        add(f"grouped_prep, {name}", like, b * (hd + 2 * kvd) * 4, 0, prep)
