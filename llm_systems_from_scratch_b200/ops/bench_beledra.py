"""Beledra at the sizes of ``bench_layers``: its configuration, and its kernels beside the like kernels of the other models, each
against its roofline (measured as ``bench_layers`` describes)."""
from __future__ import annotations

import torch

from . import mixer_ops as mo
from . import native
from .bench_layers import CONTEXT, DECODE_BATCHES, PROMPT_LEN, PROMPTS, SIZES, _bf, _expert_kernels, _residual_kernel, _Table, graph_ms, peaks
from .bench_ops import timeit

GROUP = 4                        # query heads per key/value head


def beledra_config(s: dict) -> dict:
    """Six layers over and over: matrix memory, attention twice, differential attention, matrix memory, differential attention with
    the keys and values of the one before; a dense feed-forward of the TransformerLM's width in every layer."""
    heads, mlp, mask = s["heads"], {"kind": "dense", "ff": s["ff"]}, {"size": s["window"]}
    kv = heads // GROUP
    mem = {"type": "mlstm", "mlp": mlp, "mixer": {"heads": heads, "dim": 128, "vdim": 128, "gate_cap": 15.0}}
    att = {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv, "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                                      "mask": mask, "bias_max": 1024}}
    dif = {"heads": heads, "kv_heads": kv, "dim": 64, "vdim": 128, "scale": 64 ** -0.5, "mask": mask, "diff": 0.5,
           "rot": {"base": 10000.0, "dims": 64, "scaling": {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}}}
    layers = []
    for i in range(s["runs"]):
        kind = i % 6
        if kind in (0, 4):
            layers.append(mem)
        elif kind in (1, 2):
            layers.append(att)
        else:
            layers.append({"type": "attention_2", "mlp": mlp, "mixer": {**dif, "kv_from": i - 2} if kind == 5 else dif})
    return {"architecture": "Beledra", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6}, "layers": layers}


def _shapes(s):
    """Grouped attention with a distance bias, and with two maps."""
    heads, kv, win = s["heads"], s["heads"] // GROUP, s["window"]
    bias = torch.randn(heads, min(win, 1024), device="cuda")
    return (mo.AttentionShape(heads, kv, 1, 128, 128, 0, 128 ** -0.5, win, 1e-6, bias=bias),
            mo.AttentionShape(heads, kv, 2, 64, 128, 64, 64 ** -0.5, win, 1e-6, difference=0.5, out_scale=0.5))


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
    from . import attention
    w, heads, rows, ff = s["width"], s["heads"], PROMPTS * PROMPT_LEN, s["ff"]
    hd, win = heads * 128, s["window"]
    cu = torch.arange(PROMPTS + 1, dtype=torch.int32, device="cuda") * PROMPT_LEN
    pos = torch.arange(PROMPT_LEN, dtype=torch.int32, device="cuda").repeat(PROMPTS)
    slots = torch.arange(rows, device="cuda")
    tables = torch.arange(rows // 64, device="cuda").int().view(PROMPTS, PROMPT_LEN // 64)
    seen = PROMPTS * (win * (win + 1) / 2 + (PROMPT_LEN - win) * win)
    # attention over keys
    qkv = _bf(rows, 3 * hd)
    pairs = PROMPTS * PROMPT_LEN * (PROMPT_LEN + 1) / 2
    t.add("flash_varlen_fwd (TransformerLM)", "-", timeit(lambda: attention.varlen_attention_fwd(qkv, cu, PROMPT_LEN, heads)),
          rows * hd * 8, 4 * pairs * hd)
    q, kv, gate, o = _bf(rows, hd), _bf(rows, 2 * hd), _bf(rows, hd), _bf(rows, hd)
    t.add(f"flash_window_fwd, window {win}, gate (Tedirax)", "-",
          timeit(lambda: mo.window_attention(q, kv, cu, cu, PROMPT_LEN, heads, 128, 128, win, 128 ** -0.5, o, gate)),
          rows * hd * 10, 4 * seen * hd)
    del qkv, q, kv
    for name, a in zip(("distance bias", "two maps, gate"), _shapes(s)):
        q, cache = _bf(rows, heads * a.maps * a.q_pitch), _bf(rows // 64, 64, a.cache_width)
        g = gate if a.maps == 2 else None
        t.add(f"grouped_prefill, window {win}, {name}", "flash_window_fwd",
              timeit(lambda: mo.attention_portions(q, a, cache, pos, cu, PROMPT_LEN, tables, o, g)),
              rows * (q.shape[1] + a.cache_width + hd * (2 if g is not None else 1)) * 2, 2 * seen * heads * a.maps * (a.dim + a.vdim))
    del q, cache, gate, o
    # matrix memory; the algorithms' work counted for chunks of 128 without the hi / lo parts
    proj, y = _bf(rows, 4 * hd), _bf(rows, hd)
    decay = [1.0 - 2.0 ** (-5.0 - 4.0 * i / max(1, heads - 1)) for i in range(heads)]
    powers, table = mo.retention_powers(decay, "cuda"), torch.randn(2, PROMPT_LEN, 64, device="cuda")
    seqs = torch.arange(PROMPTS, dtype=torch.int32, device="cuda")
    work = rows * heads * (4 * 128 * 128 / 2 + 4 * 128 * 128)
    state = torch.zeros(PROMPTS, heads, 128, 128, device="cuda")
    t.add("retention_chunk (Tedirax)", "-",
          timeit(lambda: mo.retention_chunked(proj, state, seqs, cu, pos, table, powers, heads, 128, 128, 128, 1e-6, y)), rows * hd * 10, work)
    state = torch.zeros(PROMPTS, heads, mo.mlstm_state(128, 128), device="cuda")
    gates, bias, nw = torch.randn(rows, 2 * heads, device="cuda"), torch.zeros(2 * heads, device="cuda"), torch.ones(hd, device="cuda").bfloat16()
    t.add("mlstm_chunk", "retention_chunk",
          timeit(lambda: mo.mlstm(proj, gates, bias, nw, state, seqs, cu, None, pos, heads, 128, 128, 15.0, 1e-6, y, True)),
          rows * hd * 10 + gates.numel() * 4, work)
    del proj, y, gates
    # products
    a, res, nw = _bf(rows, w), _bf(rows, w), torch.ones(w, device="cuda").bfloat16()
    wgu, wif = _bf(2 * ff, w), _bf(2 * heads, w)
    gu = torch.empty(rows, 2 * ff, dtype=torch.bfloat16, device="cuda")
    t.add("gate|up GEMM (TransformerLM)", "-", timeit(lambda: native.gemm(a, wgu, "nt", out=gu)),
          (rows * w + 2 * ff * w + rows * 2 * ff) * 2, 4.0 * rows * w * ff)
    t.add("silu_mul (TransformerLM)", "-", timeit(lambda: native.silu_mul_fwd(gu)), rows * ff * 6)
    del gu
    _expert_kernels(s, t, rows, torch.randint(0, s["vocab"], (rows,), device="cuda"))
    t.add("gate|up GEMM + ReLU", "experts gate|up", timeit(lambda: mo.glu(a, wgu, ff, "relu")),
          (rows * w + 2 * ff * w + rows * ff) * 2, 4.0 * rows * w * ff)
    t.add("gates GEMM (fp32 out)", "-", timeit(lambda: mo.linear(a, wif, out_dtype=torch.float32)),
          (rows * w + wif.numel()) * 2 + rows * 2 * heads * 4, 2.0 * rows * w * 2 * heads)
    # rows
    t.add("rmsnorm_fwd (TransformerLM)", "-", timeit(lambda: native.rmsnorm_fwd(res, nw, 1e-6)), rows * w * 4)
    _residual_kernel(s, t, rows)
    x = torch.randn(rows, w, device="cuda")
    t.add("add_normed", "residual_norm", timeit(lambda: mo.add_normed(x, res, nw, 1e-6)), rows * w * 12)
    pr = _bf(rows, s["q_rank"] + s["kv_rank"] + hd)
    nq, nkv = _bf(s["q_rank"]), _bf(s["kv_rank"])
    cache = torch.zeros(rows // 64, 64, s["kv_rank"], dtype=torch.bfloat16, device="cuda")
    t.add("latent_norm_append (Tedirax)", "-", timeit(lambda: mo.latent_norm_append(pr, nq, nkv, 1e-6, cache, slots)),
          rows * (s["q_rank"] + s["kv_rank"]) * 4)
    del pr, cache, x, res
    for name, a in zip(("norm", "norm, rotation"), _shapes(s)):
        n = (a.heads + a.kv_heads) * a.maps * a.dim + a.kv_heads * a.vdim
        pr, nw = _bf(rows, n + (hd if a.maps == 2 else 0)), torch.ones(a.dim, device="cuda").bfloat16()
        cache = torch.zeros(rows // 64, 64, a.cache_width, dtype=torch.bfloat16, device="cuda")
        cs = torch.randn(2, PROMPT_LEN, a.rot // 2, device="cuda") if a.rot else None
        t.add(f"grouped_prep, {name}", "latent_norm_append", timeit(lambda: mo.attention_prepare(pr, a, nw, nw, cs, pos, slots, cache)), rows * n * 4)


def _decode_kernels(s, t, b):
    from . import serving_ops
    w, heads, ff = s["width"], s["heads"], s["ff"]
    hd, win, kvr = heads * 128, min(s["window"], CONTEXT), s["kv_rank"]
    ctx = torch.full((b,), CONTEXT, dtype=torch.int32, device="cuda")
    pos, slots = ctx - 1, torch.zeros(b, dtype=torch.int64, device="cuda")

    def add(name, like, nbytes, flops, make):
        t.add(f"{name}, batch {b}", like, graph_ms(make, nbytes), nbytes, flops)
        torch.cuda.empty_cache()

    def tables(page, width):
        n = -(-(CONTEXT + 16) // page)
        tb = torch.zeros(b, width, dtype=torch.int32, device="cuda")
        tb[:, :n] = torch.randperm(b * n, device="cuda").int().view(b, n)
        return tb, b * n

    def paged():
        tb, pages = tables(16, 128)
        qkv, kc, vc = _bf(b, 3 * hd), _bf(pages, 16, hd), _bf(pages, 16, hd)
        return lambda: serving_ops.paged_decode_attention(qkv, kc, vc, tb, ctx, heads)
    add("paged_decode (TransformerLM)", "-", b * CONTEXT * hd * 4, 0, paged)

    def latent():
        tb, pages = tables(64, 32)
        ql, cache = _bf(b, heads * kvr), _bf(pages, 64, kvr)
        return lambda: mo.latent_decode(ql, cache, pos, slots, tb, heads, s["window"], 0.1)
    add(f"latent_decode, window {win} (Tedirax)", "-", b * (win * kvr * 2 + heads * kvr * 4), 4.0 * b * heads * win * kvr, latent)
    for name, a in zip(("distance bias", "two maps, gate"), _shapes(s)):
        def grouped():
            tb, pages = tables(64, 32)
            q, cache, o = _bf(b, heads * a.maps * a.q_pitch), _bf(pages, 64, a.cache_width), _bf(b, hd)
            g = _bf(b, hd) if a.maps == 2 else None
            return lambda: mo.attention_decode(q, a, cache, pos, slots, tb, o, g)
        add(f"grouped_decode, window {win}, {name}", "latent_decode", b * (win * a.cache_width + heads * a.maps * a.q_pitch + hd) * 2, 0, grouped)
    table, decay = torch.randn(2, 2048, 64, device="cuda"), torch.full((heads,), 0.99, device="cuda")

    def retention():
        state, sl = torch.randn(b, heads, 128, 128, device="cuda"), torch.randperm(b, device="cuda").int()
        proj, y = _bf(b, 4 * hd), _bf(b, hd)
        return lambda: mo.retention(proj, state, sl, None, None, pos, table, decay, heads, 128, 128, 128, 1e-6, y)
    add("retention step (Tedirax)", "-", b * heads * 128 * 128 * 8, 0, retention)
    bias, nw = torch.zeros(2 * heads, device="cuda"), torch.ones(hd, device="cuda").bfloat16()

    def memory():
        state, sl = torch.randn(b, heads, mo.mlstm_state(128, 128), device="cuda"), torch.randperm(b, device="cuda").int()
        proj, y, gates = _bf(b, 4 * hd), _bf(b, hd), (_bf(b, w), _bf(2 * heads, w))
        return lambda: mo.mlstm(proj, gates, bias, nw, state, sl, None, None, pos, heads, 128, 128, 15.0, 1e-6, y)
    add("mlstm step with gates", "retention step", b * heads * 128 * 129 * 8 + 2 * heads * w * 2, 0, memory)

    def plain(n, k):
        def make():
            a, wt = _bf(b, k), _bf(n, k)
            return lambda: mo.linear(a, wt)
        return make
    size = lambda n, k: (n * k + b * (n + k)) * 2
    kvd = heads // GROUP * 128
    for name, like, n, k in (("qkv GEMM (TransformerLM)", "-", 3 * hd, w), ("output GEMM", "-", w, hd),
                             ("gate|up GEMM (TransformerLM)", "-", 2 * ff, w), ("down GEMM", "-", w, ff),
                             ("memory q|k|v|g GEMM", "qkv GEMM", 4 * hd, w), ("attention q|k|v GEMM", "qkv GEMM", hd + 2 * kvd, w),
                             ("differential q|k|v|g GEMM", "qkv GEMM", 2 * hd + 2 * kvd, w)):
        add(name, like, size(n, k), 0, plain(n, k))

    def gate_up():
        a, wt = _bf(b, w), _bf(2 * ff, w)
        return lambda: mo.glu(a, wt, ff, "relu")
    add("gate|up GEMM + ReLU", "gate|up GEMM", (2 * ff * w + b * (w + ff)) * 2, 0, gate_up)
    nw1 = torch.ones(w, device="cuda").bfloat16()

    def norm():
        x = _bf(b, w)
        return lambda: native.rmsnorm_fwd(x, nw1, 1e-6)
    add("rmsnorm_fwd (TransformerLM)", "-", b * w * 4, 0, norm)

    def resid():
        x, y = torch.randn(b, w, device="cuda"), _bf(b, w)
        return lambda: mo.add_normed(x, y, nw1, 1e-6)
    add("add_normed", "rmsnorm_fwd", b * w * 12, 0, resid)
    nq, nkv = _bf(s["q_rank"]), _bf(kvr)

    def append():
        pr, cache = _bf(b, s["q_rank"] + kvr + hd), _bf(b, 16, kvr)
        sl = torch.arange(b, device="cuda") * 16
        return lambda: mo.latent_norm_append(pr, nq, nkv, 1e-6, cache, sl)
    add("latent_norm_append (Tedirax)", "-", b * (s["q_rank"] + kvr) * 4, 0, append)
    for name, a in zip(("norm", "norm, rotation"), _shapes(s)):
        n = (a.heads + a.kv_heads) * a.maps * a.dim + a.kv_heads * a.vdim
        nw2 = torch.ones(a.dim, device="cuda").bfloat16()
        cs = torch.randn(2, 2048, a.rot // 2, device="cuda") if a.rot else None

        def prep():
            pr, cache = _bf(b, n), _bf(b, 16, a.cache_width)
            sl = torch.arange(b, device="cuda") * 16
            return lambda: mo.attention_prepare(pr, a, nw2, nw2, cs, pos, sl, cache)
        add(f"grouped_prep, {name}", "latent_norm_append", b * n * 4, 0, prep)
