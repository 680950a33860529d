"""Throughput of the layered decoders beside the TransformerLM at equal size, and the kernels of both against their roofline.

``models(size)`` times whole steps through the serving engine (a prompt step of several prompts; a decode step at a batch
and a context), on the device with CUDA events; every step streams weights and caches that are larger than L2.
``kernels(size)`` times each kernel alone on one layer's shapes: achieved bytes or FLOPs per second over the measured copy
bandwidth or GEMM throughput.  Prompt kernels: one launch between two events, L2 replaced between runs.  Decode kernels,
which are as short as a launch: a CUDA graph of launches on different inputs that exceed L2 together, divided by their
number.  Weights are random."""
from __future__ import annotations

import gc
import json
import os

import torch

from . import mixer_ops as mo
from . import native
from .bench_ops import timeit

SIZES = {
    # width, heads of 128, TransformerLM layers / ff; the layered model has as many layer runs and twice-chosen experts whose
    # active width is the TransformerLM's ff
    "0.35b": dict(width=1024, heads=8, runs=24, ff=2816, vocab=32768, q_rank=512, kv_rank=256, window=512, distinct=12),
    "1.3b": dict(width=2048, heads=16, runs=24, ff=5504, vocab=50257, q_rank=1024, kv_rank=512, window=1024, distinct=12),
    "7b-8layers": dict(width=4096, heads=32, runs=8, ff=11008, vocab=32000, q_rank=1536, kv_rank=512, window=1024, distinct=8),
}
EXPERTS, TOP = 8, 2
PROMPTS, PROMPT_LEN = 8, 2048
DECODE_BATCHES, CONTEXT = (32, 128), 1200


def layered_config(s: dict) -> dict:
    """Three retention layers to one latent-attention layer."""
    mlp = {"kind": "moe", "expert": {"ff": s["ff"] // TOP}, "router": {"experts": EXPERTS, "top": TOP}}
    decay = [1.0 - 2.0 ** (-5.0 - 4.0 * i / max(1, s["heads"] - 1)) for i in range(s["heads"])]
    ret = {"type": "retention", "mlp": mlp, "mixer": {"heads": s["heads"], "dim": 128, "vdim": 128, "decay": decay,
                                                      "rot": {"base": 10000.0, "dims": 128}}}
    lat = {"type": "latent_attention", "mlp": mlp,
           "mixer": {"heads": s["heads"], "dim": 128, "vdim": 128, "q_rank": s["q_rank"], "kv_rank": s["kv_rank"],
                     "scale": 128 ** -0.5, "mask": {"size": s["window"]}}}
    return {"architecture": "Tedirax", "vocab": s["vocab"], "width": s["width"], "norm": {"eps": 1e-6},
            "layers": [lat if i % 4 == 3 else ret for i in range(s["distinct"])],
            "loop": {"start": 0, "stop": s["distinct"], "times": s["runs"] // s["distinct"]}}


def peaks() -> dict:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            p = json.load(f)
        return {"hbm_gbs": float(p["hbm_gbs"]), "tflops": float(p["bf16_tflops"]), "of": "measured"}
    except (OSError, KeyError, ValueError):
        return {"hbm_gbs": 6650.0, "tflops": 1590.0, "of": "fallback"}


def build(kind: str, s: dict):
    from ..models.registry import build_model
    if kind == "Tedirax":
        return build_model(layered_config(s))
    if kind == "Beledra":
        from .bench_beledra import beledra_config
        return build_model(beledra_config(s))
    if kind == "Genedra":
        from .bench_genedra import genedra_config
        return build_model(genedra_config(s))
    if kind == "Vilosun":
        from .bench_vilosun import vilosun_config
        return build_model(vilosun_config(s))
    return build_model(dict(vocab_size=s["vocab"], context_length=4096, d_model=s["width"], num_layers=s["runs"],
                            num_heads=s["heads"], d_ff=s["ff"], rope_theta=10000.0))


def step_times(kind: str, s: dict, steps: int, warmup: int) -> dict:
    """Milliseconds of one prompt step and of one decode step (graph replay) through the engine."""
    from ..serving import Request, ServingEngine
    from ..serving.batch import StepBatch
    model = build(kind, s)
    rec = {}
    g = torch.Generator().manual_seed(1)
    ids = lambda n: torch.randint(0, s["vocab"], (n,), generator=g).tolist()
    eng = ServingEngine(model, num_pages=PROMPTS * PROMPT_LEN // 16, max_batch=PROMPTS, max_context=PROMPT_LEN,
                        max_prefill_tokens=PROMPTS * PROMPT_LEN)
    reqs = [Request(i, ids(PROMPT_LEN), 0) for i in range(PROMPTS)]
    for r in reqs:
        eng.sched.open(r)
        eng.sched.grow(r, PROMPT_LEN)
    batch = StepBatch.build([(r, 0, r.prompt) for r in reqs], eng.page_size, eng.max_pages_per_req, eng.device)
    last = torch.from_numpy(batch.last_rows()).to(eng.device)
    with torch.no_grad():
        run = lambda: eng.backend.logits(eng.backend.forward(batch), last)
        native.reset_launch_count()
        run()
        launches = native.launch_count()
        rec["prefill_ms"] = timeit(run, iters=steps, warm=warmup, flush=False)
    rec["prefill_launches"] = launches
    native.check_status()
    del eng, batch
    for b in DECODE_BATCHES:
        eng = ServingEngine(model, num_pages=b * (-(-(CONTEXT + 64) // 16)) + 8, max_batch=b, max_context=2048)
        for i in range(b):
            eng.sched.add(Request(i, ids(CONTEXT), 64))
        eng._realtime, eng._virtual = False, float("inf")
        while eng.sched.waiting or eng._prefilling:
            eng.step(float("inf"))
        running = list(eng.sched.running)
        eng.decode(running)
        graph = eng._graphs[eng._bucket(b)]["graph"]
        # one event pair around several replays: a step is too short for the event's own resolution to vanish in it
        t0, t1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        for _ in range(warmup):
            graph.replay()
        torch.cuda.synchronize()
        t0.record()
        for _ in range(steps):
            graph.replay()
        t1.record()
        torch.cuda.synchronize()
        rec[f"decode_ms_b{b}"] = t0.elapsed_time(t1) / steps
        native.check_status()
        del eng, graph
        gc.collect()
        torch.cuda.empty_cache()
    del model
    gc.collect()
    torch.cuda.empty_cache()
    return rec


def models(size: str, steps: int = 10, warmup: int = 3, kinds=("Tedirax", "TransformerLM")) -> dict:
    s = SIZES[size]
    out = {"size": size, "prompts": PROMPTS, "prompt_len": PROMPT_LEN, "context": CONTEXT}
    for kind in kinds:
        rec = step_times(kind, s, steps, warmup)
        out[kind] = {"prefill_ms": round(rec["prefill_ms"], 3),
                     "prefill_tok_per_s": round(PROMPTS * PROMPT_LEN / rec["prefill_ms"] * 1e3),
                     "prefill_launches": rec["prefill_launches"],
                     **{f"decode_ms_b{b}": round(rec[f"decode_ms_b{b}"], 3) for b in DECODE_BATCHES},
                     **{f"decode_tok_per_s_b{b}": round(b / rec[f"decode_ms_b{b}"] * 1e3) for b in DECODE_BATCHES}}
    return out


class _Table:
    """Kernel records: milliseconds, and achieved bytes/s and FLOP/s as fractions of the measured peaks."""

    def __init__(self, pk):
        self.pk, self.rows = pk, []

    def add(self, name: str, like: str, ms: float, nbytes: float, flops: float = 0.0):
        roof = max(nbytes / (self.pk["hbm_gbs"] * 1e9), flops / (self.pk["tflops"] * 1e12)) * 1e3
        self.rows.append({"kernel": name, "like": like, "us": round(ms * 1e3, 1), "gb_per_s": round(nbytes / ms / 1e6),
                          "tflops": round(flops / ms / 1e9, 1), "fraction_of_roofline": round(roof / ms, 3)})


def graph_ms(make, nbytes: float) -> float:
    """Milliseconds per launch of the closures that ``make()`` returns, each on inputs of its own (``nbytes`` apiece), in one
    captured graph; together they read at least 400 MB, so nothing is found in L2 from the launch before."""
    fns = [make() for _ in range(int(max(4, min(48, 400e6 // max(1.0, nbytes) + 1))))]
    for f in fns[:2]:
        f()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    keep = []
    with torch.cuda.graph(graph):
        for f in fns:
            keep.append(f())
    return timeit(graph.replay, iters=7, warm=2, flush=True) / len(fns)


def _bf(*shape):
    return torch.randn(*shape, device="cuda").bfloat16()


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
    w, heads, rows = s["width"], s["heads"], PROMPTS * PROMPT_LEN
    hd = heads * 128
    cu = torch.arange(PROMPTS + 1, dtype=torch.int32, device="cuda") * PROMPT_LEN
    pos = torch.arange(PROMPT_LEN, dtype=torch.int32, device="cuda").repeat(PROMPTS)
    table = torch.randn(2, PROMPT_LEN, 64, device="cuda")
    # attention over keys
    qkv = _bf(rows, 3 * hd)
    pairs = PROMPTS * PROMPT_LEN * (PROMPT_LEN + 1) / 2
    t.add("flash_varlen_fwd (TransformerLM)", "-", timeit(lambda: attention.varlen_attention_fwd(qkv, cu, PROMPT_LEN, heads)),
          rows * hd * 8, 4 * pairs * hd)
    del qkv
    q, kv, gate, o = _bf(rows, hd), _bf(rows, 2 * hd), _bf(rows, hd), _bf(rows, hd)
    win = s["window"]
    seen = PROMPTS * (win * (win + 1) / 2 + (PROMPT_LEN - win) * win)
    t.add(f"flash_window_fwd, window {win}, gate", "flash_varlen_fwd",
          timeit(lambda: mo.window_attention(q, kv, cu, cu, PROMPT_LEN, heads, 128, 128, win, 128 ** -0.5, o, gate)),
          rows * hd * 10, 4 * seen * hd)
    del q, kv, gate, o
    # retention; the algorithm's work counted for chunks of 128 without the hi / lo parts
    proj, y = _bf(rows, 4 * hd), _bf(rows, hd)
    decay = [1.0 - 2.0 ** (-5.0 - 4.0 * i / max(1, heads - 1)) for i in range(heads)]
    powers = mo.retention_powers(decay, "cuda")
    state = torch.zeros(PROMPTS, heads, 128, 128, device="cuda")
    slots = torch.arange(PROMPTS, dtype=torch.int32, device="cuda")
    t.add("retention_chunk", "flash_varlen_fwd",
          timeit(lambda: mo.retention_chunked(proj, state, slots, cu, pos, table, powers, heads, 128, 128, 128, 1e-6, y)),
          rows * hd * 10, rows * heads * (4 * 128 * 128 / 2 + 4 * 128 * 128))
    del proj, y
    # products
    a, wd = _bf(rows, w), _bf(2 * s["ff"], w)
    gu = torch.empty(rows, 2 * s["ff"], dtype=torch.bfloat16, device="cuda")
    t.add("gate|up GEMM (TransformerLM)", "-", timeit(lambda: native.gemm(a, wd, "nt", out=gu)),
          (rows * w + 2 * s["ff"] * w + rows * 2 * s["ff"]) * 2, 4.0 * rows * w * s["ff"])
    t.add("silu_mul (TransformerLM)", "-", timeit(lambda: native.silu_mul_fwd(gu)), rows * s["ff"] * 6)
    h, dn = _bf(rows, s["ff"]), _bf(w, s["ff"])
    res = _bf(rows, w)
    t.add("down GEMM + residual (TransformerLM)", "-", timeit(lambda: native.gemm(h, dn, "nt", residual=res)),
          (rows * s["ff"] + s["ff"] * w + 2 * rows * w) * 2, 2.0 * rows * w * s["ff"])
    del gu, h, wd
    _expert_kernels(s, t, rows, torch.randint(0, s["vocab"], (rows,), device="cuda"))
    # residual stream
    nw = torch.ones(w, device="cuda").bfloat16()
    t.add("rmsnorm_fwd (TransformerLM)", "-", timeit(lambda: native.rmsnorm_fwd(res, nw, 1e-6)), rows * w * 4)
    _residual_kernel(s, t, rows)
    # latents
    pr = _bf(rows, s["q_rank"] + s["kv_rank"] + hd)
    nq, nkv = _bf(s["q_rank"]), _bf(s["kv_rank"])
    cache = torch.zeros(rows // 64, 64, s["kv_rank"], dtype=torch.bfloat16, device="cuda")
    sl = torch.randperm(rows, device="cuda")
    t.add("latent_norm_append", "rmsnorm_fwd", timeit(lambda: mo.latent_norm_append(pr, nq, nkv, 1e-6, cache, sl)),
          rows * (s["q_rank"] + s["kv_rank"]) * 4)
    tables = torch.randperm(rows // 64, device="cuda").int().view(PROMPTS, PROMPT_LEN // 64)
    first = torch.zeros(PROMPTS, dtype=torch.int32, device="cuda")
    del cache

    def gather():
        c = torch.zeros(rows // 64, 64, s["kv_rank"], dtype=torch.bfloat16, device="cuda")
        return lambda: mo.latent_gather(c, cu, first, tables, rows)
    t.add("latent_gather", "rmsnorm_fwd", graph_ms(gather, rows * s["kv_rank"] * 4), rows * s["kv_rank"] * 4)


def _expert_kernels(s, t, rows, tokens):
    w, ff = s["width"], s["ff"] // TOP
    table = torch.rand(s["vocab"], EXPERTS, device="cuda").argsort(1)[:, :TOP].int().contiguous()
    live = torch.zeros(rows, dtype=torch.int64, device="cuda")
    layers = 12
    ms = timeit(lambda: mo.moe_plan(tokens, live, [table] * layers, [EXPERTS] * layers))
    t.add(f"moe_plan, {layers} layers, {rows} rows", "-", ms, layers * rows * TOP * 8)
    pos, groups = mo.moe_plan(tokens, live, [table], [EXPERTS])
    p = mo.plan_tiles(rows, EXPERTS, TOP) * mo.TILE
    xg = _bf(p, w)
    w_gu, w_dn = _bf(EXPERTS * 2 * ff, w), _bf(EXPERTS * w, ff)
    n = rows * TOP
    active = min(EXPERTS, n)
    hid = mo.gemm_rows(xg, w_gu, groups[0], ff, True)
    t.add(f"experts gate|up + SwiGLU, {rows} rows", "gate|up GEMM", timeit(lambda: mo.gemm_rows(xg, w_gu, groups[0], ff, True)),
          (n * w + active * 2 * ff * w + n * ff) * 2, 4.0 * n * w * ff)
    t.add(f"experts down, {rows} rows", "down GEMM", timeit(lambda: mo.gemm_rows(hid, w_dn, groups[0], w, False)),
          (n * ff + active * ff * w + n * w) * 2, 2.0 * n * w * ff)


def _residual_kernel(s, t, rows):
    w = s["width"]
    x = torch.randn(rows, w, device="cuda")
    p = mo.plan_tiles(rows, EXPERTS, TOP) * mo.TILE
    y = _bf(p, w)
    perm = torch.randperm(p, device="cuda")[:rows * TOP].int().view(rows, TOP).contiguous()
    nw = torch.ones(w, device="cuda").bfloat16()
    t.add(f"residual_norm with experts, {rows} rows", "rmsnorm_fwd",
          timeit(lambda: mo.residual_norm(x, nw, 1e-6, pending=(y, perm, 0.0), scatter=(perm, p))),
          rows * w * (8 + 2 * TOP + 2 + 2 * TOP))


def _decode_kernels(s, t, b):
    from . import serving_ops
    w, heads = s["width"], s["heads"]
    hd = heads * 128
    pages = -(-(CONTEXT + 16) // 16)
    ctx = torch.full((b,), CONTEXT, dtype=torch.int32, device="cuda")
    pos, slots = ctx - 1, torch.zeros(b, dtype=torch.int64, device="cuda")
    kvr, win = s["kv_rank"], min(s["window"], CONTEXT)

    def tables():
        full = torch.zeros(b, 128, dtype=torch.int32, device="cuda")
        full[:, :pages] = torch.randperm(b * pages, device="cuda").int().view(b, pages)
        return full

    def add(name, like, nbytes, flops, make):
        t.add(f"{name}, batch {b}", like, graph_ms(make, nbytes), nbytes, flops)
        torch.cuda.empty_cache()

    def paged():
        qkv, kc, vc, tb = _bf(b, 3 * hd), _bf(b * pages, 16, hd), _bf(b * pages, 16, hd), tables()
        return lambda: serving_ops.paged_decode_attention(qkv, kc, vc, tb, ctx, heads)
    add("paged_decode (TransformerLM)", "-", b * CONTEXT * hd * 4, 0, paged)

    def latent():
        n = -(-pages // 4)                            # pages of 64 tokens
        tb = torch.zeros(b, 32, dtype=torch.int32, device="cuda")
        tb[:, :n] = torch.randperm(b * n, device="cuda").int().view(b, n)
        ql, cache = _bf(b, heads * kvr), _bf(b * n, 64, kvr)
        return lambda: mo.latent_decode(ql, cache, pos, slots, tb, heads, s["window"], 0.1)
    add(f"latent_decode, window {win}", "paged_decode", b * (win * kvr * 2 + heads * kvr * 4), 4.0 * b * heads * win * kvr, latent)
    table, decay = torch.randn(2, 2048, 64, device="cuda"), torch.full((heads,), 0.99, device="cuda")

    def step():
        state, sl = torch.randn(b, heads, 128, 128, device="cuda"), torch.randperm(b, device="cuda").int()
        proj, y = _bf(b, 4 * hd), _bf(b, hd)
        return lambda: mo.retention(proj, state, sl, None, None, pos, table, decay, heads, 128, 128, 128, 1e-6, y)
    add("retention step", "paged_decode", b * heads * 128 * 128 * 8, 0, step)

    def plain(n, k):
        def make():
            a, wt = _bf(b, k), _bf(n, k)
            return lambda: mo.linear(a, wt)
        return make
    size = lambda n, k: (n * k + b * (n + k)) * 2
    for name, like, n, k in (("qkv GEMM (TransformerLM)", "-", 3 * hd, w), ("output GEMM (TransformerLM)", "-", w, hd),
                             ("gate|up GEMM (TransformerLM)", "-", 2 * s["ff"], w), ("down GEMM (TransformerLM)", "-", w, s["ff"]),
                             ("retention q|k|v|g GEMM", "qkv GEMM", 4 * hd, w),
                             ("latent dq|dkv|g GEMM", "qkv GEMM", s["q_rank"] + kvr + hd, w), ("latent uq GEMM", "output GEMM", hd, s["q_rank"])):
        add(name, like, size(n, k), 0, plain(n, k))

    def out_gemm():
        a, wt, x = _bf(b, hd), _bf(w, hd), torch.zeros(b, w, device="cuda")
        return lambda: mo.linear(a, wt, out=x, accumulate=True)
    add("output GEMM into the fp32 residual", "output GEMM", (w * hd + b * hd) * 2 + b * w * 8, 0, out_gemm)

    def to_latent():
        q, wk = _bf(b, hd), _bf(heads * kvr, 128)
        return lambda: mo.gemm_heads(q, wk, heads, 128, kvr)
    add("queries into latent space", "output GEMM", (heads * kvr * 128 + b * hd + b * heads * kvr) * 2, 0, to_latent)

    def from_latent():
        ol, wv, gate = _bf(b, heads * kvr), _bf(hd, kvr), _bf(b, hd)
        return lambda: mo.gemm_heads(ol, wv, heads, kvr, 128, gate=gate)
    add("latent outputs to heads, gate", "output GEMM", (heads * kvr * 128 + 2 * b * hd + b * heads * kvr) * 2, 0, from_latent)
    ff, n = s["ff"] // TOP, b * TOP
    tab = torch.rand(s["vocab"], EXPERTS, device="cuda").argsort(1)[:, :TOP].int().contiguous()
    tokens = torch.randint(0, s["vocab"], (b,), device="cuda")
    add("moe_plan, 12 layers", "-", 12 * n * 8, 0, lambda: (lambda: mo.moe_plan(tokens, slots, [tab] * 12, [EXPERTS] * 12)))
    (mpos,), (group,) = mo.moe_plan(tokens, slots, [tab], [EXPERTS])
    p, active = mo.plan_tiles(b, EXPERTS, TOP) * mo.TILE, min(EXPERTS, n)

    def gate_up():
        xg, wt = _bf(p, w), _bf(EXPERTS * 2 * ff, w)
        return lambda: mo.gemm_rows(xg, wt, group, ff, True)
    add("experts gate|up + SwiGLU", "gate|up GEMM", (n * w + active * 2 * ff * w + n * ff) * 2, 4.0 * n * w * ff, gate_up)

    def down():
        hid, wt = _bf(p, ff), _bf(EXPERTS * w, ff)
        return lambda: mo.gemm_rows(hid, wt, group, w, False)
    add("experts down", "down GEMM", (n * ff + active * ff * w + n * w) * 2, 2.0 * n * w * ff, down)
    nw = torch.ones(w, device="cuda").bfloat16()

    def resid():
        x, y = torch.randn(b, w, device="cuda"), _bf(p, w)
        return lambda: mo.residual_norm(x, nw, 1e-6, pending=(y, mpos, 0.0), scatter=(mpos, p))
    add("residual_norm with experts", "rmsnorm_fwd", b * w * (8 + 2 * TOP + 2 + 2 * TOP), 0, resid)

    def norm():
        x = _bf(b, w)
        return lambda: native.rmsnorm_fwd(x, nw, 1e-6)
    add("rmsnorm_fwd (TransformerLM)", "-", b * w * 4, 0, norm)
    nq, nkv = _bf(s["q_rank"]), _bf(kvr)

    def append():
        pr, cache = _bf(b, s["q_rank"] + kvr + hd), _bf(b, 16, kvr)
        sl = torch.arange(b, device="cuda") * 16
        return lambda: mo.latent_norm_append(pr, nq, nkv, 1e-6, cache, sl)
    add("latent_norm_append", "rmsnorm_fwd", b * (s["q_rank"] + kvr) * 4, 0, append)


def run(sizes, steps: int = 10, warmup: int = 3, per_kernel: bool = True, model: str = "Tedirax"):
    """One record per size: Tedirax beside the TransformerLM, Beledra beside both, Genedra or Vilosun beside the models before it."""
    for size in sizes:
        if model == "Beledra":
            from . import bench_beledra
            rec = models(size, steps, warmup, ("Beledra", "Tedirax", "TransformerLM"))
            more = bench_beledra.kernels
        elif model == "Genedra":
            from . import bench_genedra
            rec = models(size, steps, warmup, ("Genedra", "Tedirax", "Beledra", "TransformerLM"))
            more = bench_genedra.kernels
        elif model == "Vilosun":
            from . import bench_vilosun
            rec = models(size, steps, warmup, ("Vilosun", "Tedirax", "Beledra", "Genedra", "TransformerLM"))
            more = bench_vilosun.kernels
        else:
            rec, more = models(size, steps, warmup), kernels
        if per_kernel:
            rec.update(more(size))
        yield rec
