"""Vilosun at the sizes of ``bench_layers``: its configuration, and its kernels beside the like kernels of the other models, each
against its roofline (measured as ``bench_layers`` describes)."""
from __future__ import annotations

import torch

from . import mixer_ops as mo
from . import native
from .bench_layers import (CONTEXT, DECODE_BATCHES, EXPERTS, PROMPT_LEN, PROMPTS, SIZES, TOP, _bf, _expert_kernels, _residual_kernel,
                           _Table, graph_ms, peaks)
from .bench_ops import timeit

GROUP, SHARED = 4, 2             # query heads per key/value head (attention), heads per key (delta rule)
TAPS, ATTENTION_TAPS, GROUPS = 4, 3, 8


def vilosun_config(s: dict) -> dict:
    """Three delta rules to one attention, two of eight experts in every layer whose active width is the TransformerLM's."""
    heads = s["heads"]
    moe = {"kind": "moe", "expert": {"ff": s["ff"] // TOP}, "router": {"experts": EXPERTS, "top": TOP}}
    rule = {"type": "delta", "mlp": moe, "mixer": {"heads": heads, "kv_heads": heads // SHARED, "dim": 128, "vdim": 128, "conv": TAPS}}
    att = {"type": "attention", "mlp": moe, "mixer": {"heads": heads, "kv_heads": heads // GROUP, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                                      "conv": ATTENTION_TAPS, "mask": {"size": s["window"]}, "v_mix": True}}
    return {"architecture": "Vilosun", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6, "groups": GROUPS}, "logit_scale": 0.125,
            "embedding": {"scale": 8.0, "bigram": {"buckets": 50021, "mul_prev": 50261, "mul_cur": 1}},
            "layers": [att if i % 4 == 3 else rule for i in range(s["runs"])]}


def _grouped(s):
    """Beledra's attention with a distance bias, and Vilosun's."""
    heads, kv, win = s["heads"], s["heads"] // GROUP, s["window"]
    bias, slopes = torch.randn(heads, min(win, 1024), device="cuda"), torch.tensor([2.0 ** (-8 * (h + 1) / heads) for h in range(heads)], device="cuda")
    return (mo.AttentionShape(heads, kv, 1, 128, 128, 0, 128 ** -0.5, win, 1e-6, bias=bias),
            mo.AttentionShape(heads, kv, 1, 128, 128, 0, 128 ** -0.5, win, 1e-6, slopes=slopes, chunked=True, head_gate=True))


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


def _rule(heads):
    """Parameters of a delta rule: decay, dt, head norm."""
    return -torch.rand(heads, device="cuda"), torch.randn(heads, device="cuda") - 2.0, torch.ones(128, device="cuda").bfloat16()


def _prompt_kernels(s, t):
    w, heads, rows, ff = s["width"], s["heads"], PROMPTS * PROMPT_LEN, s["ff"]
    hd, win, kv, kd = heads * 128, s["window"], heads // GROUP, heads // SHARED * 128
    cu = torch.arange(PROMPTS + 1, dtype=torch.int32, device="cuda") * PROMPT_LEN
    pos = torch.arange(PROMPT_LEN, dtype=torch.int32, device="cuda").repeat(PROMPTS)
    slots, seqs = torch.arange(rows, device="cuda"), torch.arange(PROMPTS, dtype=torch.int32, device="cuda")
    at = mo.StepRows(pos, slots, seqs, seqs.repeat_interleave(PROMPT_LEN).contiguous(), 0, cu, [])
    tables = torch.arange(rows // 64, device="cuda").int().view(PROMPTS, PROMPT_LEN // 64)
    seen, chunked = PROMPTS * (win * (win + 1) / 2 + (PROMPT_LEN - win) * win), PROMPTS * (PROMPT_LEN // win) * (win * (win + 1) / 2)
    # attention over keys
    o, hg = _bf(rows, hd), _bf(rows, heads)
    for name, like, a, pairs, g in zip(("window, distance bias (Beledra)", "chunks, slopes, gate per head"), ("-", "grouped_prefill, distance bias"),
                                       _grouped(s), (seen, chunked), (None, hg)):
        q, cache = _bf(rows, heads * a.q_pitch), _bf(rows // 64, 64, a.cache_width)
        t.add(f"grouped_prefill, {win}, {name}", like, timeit(lambda: mo.attention_portions(q, a, cache, pos, cu, PROMPT_LEN, tables, o, g)),
              rows * (q.shape[1] + a.cache_width + hd) * 2, 4 * pairs * hd)
    del q, cache, o
    # recurrences; the algorithms' work counted for chunks of 128 (retention, mLSTM) and 64 (delta rule) without the hi / lo parts
    proj, y = _bf(rows, 4 * hd), _bf(rows, hd)
    decay = [1.0 - 2.0 ** (-5.0 - 4.0 * i / max(1, heads - 1)) for i in range(heads)]
    powers, table = mo.retention_powers(decay, "cuda"), torch.randn(2, PROMPT_LEN, 64, device="cuda")
    work = rows * heads * 6 * 128 * 128
    state = torch.zeros(PROMPTS, heads, 128, 128, device="cuda")
    t.add("retention_chunk (Tedirax)", "-",
          timeit(lambda: mo.retention_chunked(proj, state, seqs, cu, pos, table, powers, heads, 128, 128, 128, 1e-6, y)), rows * hd * 10, work)
    memory = torch.zeros(PROMPTS, heads, mo.mlstm_state(128, 128), device="cuda")
    gates, bias, nw = torch.randn(rows, 2 * heads, device="cuda"), torch.zeros(2 * heads, device="cuda"), torch.ones(hd, device="cuda").bfloat16()
    t.add("mlstm_chunk (Beledra)", "-", timeit(lambda: mo.mlstm(proj, gates, bias, nw, memory, seqs, cu, None, pos, heads, 128, 128, 15.0, 1e-6, y, True)),
          rows * hd * 10 + gates.numel() * 4, work)
    c, gate, params = proj[:, :2 * kd + hd], proj[:, 3 * hd:], _rule(heads)
    n = PROMPT_LEN // mo.DELTA_CHUNK
    chunks = (torch.arange(PROMPTS + 1, dtype=torch.int32, device="cuda") * n, PROMPTS * n)
    t.add("delta_prepare + delta_chunk", "mlstm_chunk", timeit(lambda: mo.delta_rule(c, gate, gates, *params, state, at, heads // SHARED, 1e-6, y, chunks=chunks)),
          rows * (2 * kd + 3 * hd) * 2 + gates.numel() * 4, rows * heads * 7 * 128 * 128)
    filt, ring = _bf(TAPS, 2 * kd + hd), _bf(PROMPTS, TAPS, 2 * kd + hd)
    out = _bf(rows, 2 * kd + hd)
    t.add("short_conv + silu", "grouped_prep", timeit(lambda: mo.short_conv(c, filt, ring, at, out, True)), rows * (2 * kd + hd) * 4)
    del proj, y, gates, c, gate, out
    for name, like, a in zip(("grouped_prep (Beledra)", "short_conv_attend, mixed values"), ("-", "grouped_prep"), _grouped(s)):
        m = (heads + 2 * kv) * 128
        pr, cache = _bf(rows, m), torch.zeros(rows // 64, 64, a.cache_width, dtype=torch.bfloat16, device="cuda")
        if a.chunked:
            filt, ring, first, temp = _bf(ATTENTION_TAPS, m), _bf(PROMPTS, ATTENTION_TAPS, m), _bf(rows // 64, 64, a.cache_width), torch.ones(heads, device="cuda")
            t.add(name, like, timeit(lambda: mo.conv_attend(pr, filt, ring, at, a, temp, cache, first, 0.5)), rows * (m * 4 + kv * 128 * 2))
        else:
            wq, wk = (torch.ones(128, device="cuda").bfloat16() for _ in range(2))
            t.add(name, like, timeit(lambda: mo.attention_prepare(pr, a, wq, wk, None, pos, slots, cache)), rows * m * 4)
    del pr, cache, first, filt, ring
    # products
    a, res = _bf(rows, w), torch.zeros(rows, w, device="cuda")
    wi, wb, bi = _bf(4 * hd, w), _bf(2 * kd + 2 * hd + w, w), torch.randn(2 * kd + 2 * hd + w, device="cuda")
    t.add("retention q|k|v|g GEMM (Tedirax)", "-", timeit(lambda: mo.linear(a, wi)), (rows * w + wi.numel() + rows * len(wi)) * 2, 2.0 * rows * wi.numel())
    t.add("delta q|k|v|g|out GEMM, bias", "retention q|k|v|g GEMM", timeit(lambda: mo.linear(a, wb, bias=bi)), (rows * w + wb.numel() + rows * len(wb)) * 2,
          2.0 * rows * wb.numel())
    wo = _bf(w, w)
    t.add("output GEMM into the fp32 residual (Tedirax)", "-", timeit(lambda: mo.linear(a, wo, out=res, accumulate=True)), (rows * w + w * w) * 2 + rows * w * 8,
          2.0 * rows * w * w)
    t.add("gate GEMM of the feed-forward, bias", "output GEMM", timeit(lambda: mo.linear(a, wo, bias=bi[:w].contiguous())), (2 * rows * w + w * w) * 2, 2.0 * rows * w * w)
    wab = _bf(2 * heads, w)
    t.add("a|b GEMM (fp32 out)", "-", timeit(lambda: mo.linear(a, wab, out_dtype=torch.float32)), (rows * w + wab.numel()) * 2 + rows * 2 * heads * 4, 2.0 * rows * wab.numel())
    del wi, wb, wo, res
    _expert_kernels(s, t, rows, torch.randint(0, s["vocab"], (rows,), device="cuda"))
    z, live, rb = torch.randn(rows, EXPERTS, device="cuda"), torch.zeros(rows, dtype=torch.int64, device="cuda"), torch.zeros(EXPERTS, device="cuda")
    zero = lambda: torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
    t.add("moe_route (Genedra)", "-", timeit(lambda: mo.moe_route(z, rb, live, EXPERTS, TOP, zero())), rows * (EXPERTS * 4 + TOP * 12))
    t.add("moe_route by logit", "moe_route", timeit(lambda: mo.moe_route(z, None, live, EXPERTS, TOP, zero(), bias=rb)), rows * (EXPERTS * 4 + TOP * 12))
    count = zero()
    choice, rank, weight = mo.moe_route(z, None, live, EXPERTS, TOP, count, bias=rb)
    _, mpos, _ = mo.moe_dispatch(a, choice, rank, count)
    # rows
    nw = torch.ones(w, device="cuda").bfloat16()
    _residual_kernel(s, t, rows)
    x, y, gate = torch.randn(rows, w, device="cuda"), _bf(rows, w), _bf(rows, w)
    t.add("add_normed (Beledra)", "-", timeit(lambda: mo.add_normed(x, y, nw, 1e-6)), rows * w * 12)
    t.add("group_step, gated output", "add_normed", timeit(lambda: mo.group_step(x, GROUPS, 1e-6, nw, sub=mo.GatedOutput(y, gate, nw))), rows * w * 14)
    ye = _bf(mo.plan_tiles(rows, EXPERTS, TOP) * mo.TILE, w)
    ex = mo.ExpertOutputs(ye, mpos, 1.0, weight)
    t.add("group_step, gated experts", "residual_norm", timeit(lambda: mo.group_step(x, GROUPS, 1e-6, nw, sub=mo.GatedOutput(ex, gate, nw))), rows * w * (12 + 2 * TOP))


def _decode_kernels(s, t, b):
    w, heads, ff = s["width"], s["heads"], s["ff"]
    hd, win, kv, kd, f = heads * 128, min(s["window"], CONTEXT), heads // GROUP, heads // SHARED * 128, ff // TOP
    pos, slots = torch.full((b,), CONTEXT - 1, dtype=torch.int32, device="cuda"), torch.zeros(b, dtype=torch.int64, device="cuda")
    seen = (CONTEXT - 1) % s["window"] + 1                       # keys of the last token's chunk
    lines = torch.arange(b, dtype=torch.int32, device="cuda")

    def add(name, like, nbytes, flops, make):
        t.add(f"{name}, batch {b}", like, graph_ms(make, nbytes), nbytes, flops)
        torch.cuda.empty_cache()

    def tables():
        n = -(-(CONTEXT + 16) // 64)
        tb = torch.zeros(b, 32, dtype=torch.int32, device="cuda")
        tb[:, :n] = torch.randperm(b * n, device="cuda").int().view(b, n)
        return tb, b * n
    full = pos - pos + s["window"] - 1                           # the longest a chunk can be
    for name, like, a, keys, p in (("window, distance bias (Beledra)", "-", _grouped(s)[0], win, pos),
                                   ("chunk, slopes, gate per head", "grouped_decode, distance bias", _grouped(s)[1], win, full),
                                   (f"chunk at context {CONTEXT}", "grouped_decode, distance bias", _grouped(s)[1], seen, pos)):
        def grouped():
            tb, pages = tables()
            q, cache, o, g = _bf(b, heads * a.q_pitch), _bf(pages, 64, a.cache_width), _bf(b, hd), _bf(b, heads) if a.head_gate else None
            return lambda: mo.attention_decode(q, a, cache, p, slots, tb, o, g)
        add(f"grouped_decode, {s['window']}, {name}", like, b * (keys * a.cache_width + heads * a.q_pitch + hd) * 2, 0, grouped)
    # recurrences
    table, decay = torch.randn(2, 2048, 64, device="cuda"), torch.full((heads,), 0.99, device="cuda")

    def retention():
        state, sl, proj, y = torch.randn(b, heads, 128, 128, device="cuda"), torch.randperm(b, device="cuda").int(), _bf(b, 4 * hd), _bf(b, hd)
        return lambda: mo.retention(proj, state, sl, None, None, pos, table, decay, heads, 128, 128, 128, 1e-6, y)
    add("retention step (Tedirax)", "-", b * heads * 128 * 128 * 8, 0, retention)

    def mlstm():
        state, sl, proj, y = torch.randn(b, heads, mo.mlstm_state(128, 128), device="cuda"), torch.randperm(b, device="cuda").int(), _bf(b, 4 * hd), _bf(b, hd)
        h, wg, bias, nw = _bf(b, w), _bf(2 * heads, w), torch.zeros(2 * heads, device="cuda"), torch.ones(hd, device="cuda").bfloat16()
        return lambda: mo.mlstm(proj, (h, wg), bias, nw, state, sl, None, None, pos, heads, 128, 128, 15.0, 1e-6, y)
    add("mlstm step with its gates (Beledra)", "-", b * heads * mo.mlstm_state(128, 128) * 8, 0, mlstm)
    channels = 2 * kd + hd

    def rule():
        state, sl, proj, y = torch.randn(b, heads, 128, 128, device="cuda"), torch.randperm(b, device="cuda").int(), _bf(b, channels + hd), _bf(b, hd)
        h, wab, filt, ring, params = _bf(b, w), _bf(2 * heads, w), _bf(TAPS, channels), _bf(b, TAPS, channels), _rule(heads)
        at = mo.StepRows(pos, slots, sl, lines, 0, None, [])
        return lambda: mo.delta_rule(proj[:, :channels], proj[:, channels:], (h, wab), *params, state, at, heads // SHARED, 1e-6, y, conv=(filt, ring))
    add("delta step with convolution and gates", "mlstm step", b * heads * 128 * 128 * 8 + b * channels * 2 * (TAPS + 1), 0, rule)
    at = torch.arange(b, device="cuda") * 16
    for name, like, a in zip(("grouped_prep (Beledra)", "short_conv_attend, mixed values"), ("-", "grouped_prep"), _grouped(s)):
        m = (heads + 2 * kv) * 128

        def prep():
            pr, cache = _bf(b, m), _bf(b, 16, a.cache_width)
            if a.chunked:
                filt, ring, first, temp = _bf(ATTENTION_TAPS, m), _bf(b, ATTENTION_TAPS, m), _bf(b, 16, a.cache_width), torch.ones(heads, device="cuda")
                rows = mo.StepRows(pos, at, lines, lines, 0, None, [])
                return lambda: mo.conv_attend(pr, filt, ring, rows, a, temp, cache, first, 0.5)
            wq, wk = (torch.ones(128, device="cuda").bfloat16() for _ in range(2))
            return lambda: mo.attention_prepare(pr, a, wq, wk, None, pos, at, cache)
        # (the convolution reads its input, the rows before it and the first values, and writes the result and its row of the ring)
        add(name, like, b * m * 4 + (b * (m * 2 * ATTENTION_TAPS + kv * 256) if a.chunked else 0), 0, prep)
    # products

    def plain(n, k, **kw):
        def make():
            x, wt = _bf(b, k), _bf(n, k)
            return lambda: mo.linear(x, wt, **kw)
        return make
    size = lambda n, k: (n * k + b * (n + k)) * 2
    bias = lambda n: {"bias": torch.randn(n, device="cuda")}
    n_rule, n_att = channels + hd + w, (heads + 2 * kv) * 128 + w + mo.pitch(heads)
    for name, like, n, k, kw in (("retention q|k|v|g GEMM (Tedirax)", "-", 4 * hd, w, {}), ("delta q|k|v|g|out GEMM, bias", "retention q|k|v|g GEMM", n_rule, w, bias(n_rule)),
                                 ("attention q|k|v|g|out GEMM, bias", "retention q|k|v|g GEMM", n_att, w, bias(n_att)),
                                 ("output GEMM (TransformerLM)", "-", w, hd, {}), ("gate GEMM of the feed-forward, bias", "output GEMM", w, w, bias(w))):
        add(name, like, size(n, k), 0, plain(n, k, **kw))
    # experts

    def route(by_logit):
        def make():
            h, wr, rb, counts = _bf(b, w), _bf(EXPERTS, w), torch.zeros(EXPERTS, device="cuda"), torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
            if by_logit:
                return lambda: mo.moe_route_rows(h, wr, None, slots, EXPERTS, TOP, counts, bias=rb)
            return lambda: mo.moe_route_rows(h, wr, rb, slots, EXPERTS, TOP, counts)
        return make
    nbytes = ((b + EXPERTS) * w + b * EXPERTS * 2 + b * TOP * 6) * 2
    add("moe_route_rows (Genedra)", "-", nbytes, 0, route(False))
    add("moe_route_rows by logit", "moe_route_rows", nbytes, 0, route(True))
    tab = torch.rand(s["vocab"], EXPERTS, device="cuda").argsort(1)[:, :TOP].int().contiguous()
    tokens = torch.randint(0, s["vocab"], (b,), device="cuda")
    (ppos,), (group,) = mo.moe_plan(tokens, slots, [tab], [EXPERTS])
    p, n = mo.plan_tiles(b, EXPERTS, TOP) * mo.TILE, b * TOP
    for name, k, width, glu in (("experts gate|up + SwiGLU", w, f, True), ("experts down", f, w, False)):
        def rows_gemm():
            xg, wt = _bf(p, k), _bf(EXPERTS * width * (2 if glu else 1), k)
            return lambda: mo.gemm_rows(xg, wt, group, width, glu)
        mats = 2 if glu else 1
        add(f"{name} (as Tedirax)", "-", (n * k + EXPERTS * mats * width * k + n * width) * 2, 2.0 * mats * n * width * k, rows_gemm)
    # rows
    nw = torch.ones(w, device="cuda").bfloat16()
    count = torch.zeros(EXPERTS, dtype=torch.int32, device="cuda")
    choice, rank, weight = mo.moe_route(torch.randn(b, EXPERTS, device="cuda"), None, slots, EXPERTS, TOP, count)
    _, mpos, _ = mo.moe_dispatch(_bf(b, w), choice, rank, count)

    def resid(kind):
        def make():
            x, y, ye, gate = torch.randn(b, w, device="cuda"), _bf(b, w), _bf(p, w), _bf(b, w)
            if kind == "tedirax":
                return lambda: mo.residual_norm(x, nw, 1e-6, pending=(ye, ppos, 0.0), scatter=(ppos, p))
            if kind == "beledra":
                return lambda: mo.add_normed(x, y, nw, 1e-6)
            ex = mo.ExpertOutputs(ye, mpos, 1.0, weight) if kind == "experts" else y
            return lambda: mo.group_step(x, GROUPS, 1e-6, nw, sub=mo.GatedOutput(ex, gate, nw))
        return make
    add("residual_norm with experts (Tedirax)", "-", b * w * (8 + 2 * TOP + 2 + 2 * TOP), 0, resid("tedirax"))
    add("group_step, gated experts", "residual_norm", b * w * (12 + 2 * TOP), 0, resid("experts"))
    add("add_normed (Beledra)", "-", b * w * 12, 0, resid("beledra"))
    add("group_step, gated output", "add_normed", b * w * 14, 0, resid("plain"))
