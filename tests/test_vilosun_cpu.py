"""Vilosun on the CPU statements of its kernels: configuration, weights, scheduling, caches and batches against the plain
oracle (the kernels themselves: tests/test_gpu_vilosun.py)."""
import json
import math
import warnings

import pytest
import torch

import vilosun_helpers as H
import vilosun_oracle as O
from llm_systems_from_scratch_b200.models.mixers import DeltaRule, GroupedAttention, RoutedExperts
from llm_systems_from_scratch_b200.models.registry import build_model, load_model, model_class
from llm_systems_from_scratch_b200.models.vilosun import RandomTensors, Vilosun, VilosunConfig, tensor_shapes
from llm_systems_from_scratch_b200.ops import mixer_ops as mo
from llm_systems_from_scratch_b200.serving import Request, ServingEngine
from llm_systems_from_scratch_b200.serving.batch import StepBatch
from llm_systems_from_scratch_b200.serving.kv_cache import LayerCache
from llm_systems_from_scratch_b200.utils import safetensors as st

CPU = dict(dtype=torch.float32, device="cpu")


def engine(cfg, ts, **kw):
    args = dict(num_pages=24, page_size=4, max_batch=3, max_context=96)
    args.update(kw)
    return ServingEngine(Vilosun(cfg, ts, **CPU), **args)


def randn(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_is_read_and_checked():
    cfg = H.CONFIGS["odd"]
    c = VilosunConfig.from_dict(cfg)
    assert [la.type for la in c.layers].count("delta") == 3 and c.first_values == 2 and c.layers[1].mlp is None
    assert (c.eps, c.groups, c.embed_scale, c.buckets, c.mul_prev, c.logit_scale) == (1e-4, 5, 1.0, 37, 40000001, 1.0)
    la = cfg["layers"]
    mix = lambda i, **kw: {**la[i], "mixer": {**la[i]["mixer"], **kw}}
    mlp = lambda i, **kw: {**la[i], "mlp": {**la[i]["mlp"], **kw}}
    bad = ([{**la[0], "type": "convolution"}], [mix(0, kv_heads=4)], [mix(1, kv_heads=4)], [mix(0, mask={"size": 0})], [mix(0, mask={})],
           [la[2], mix(4, vdim=9)], [la[2], mix(4, kv_heads=3)], [mlp(0, kind="dense")], [mlp(0, router={"experts": 5, "top": 6})],
           [mlp(0, router={"experts": 5, "top": 0})], [mlp(0, expert={})], [{"type": "delta", "mixer": {"heads": 2}}])
    for layers in bad:
        with pytest.raises(ValueError):
            VilosunConfig.from_dict({**cfg, "layers": layers})
    for key, value in (("embedding", None), ("logit_scale", None), ("norm", {"eps": 1e-5}), ("norm", {"eps": 1e-5, "groups": 7}),
                       ("embedding", {"scale": 1.0}), ("embedding", {"scale": 1.0, "bigram": {"buckets": 0, "mul_prev": 1, "mul_cur": 1}})):
        with pytest.raises(ValueError):
            VilosunConfig.from_dict({k: v for k, v in cfg.items() if k != key} | ({} if value is None else {key: value}))
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        with pytest.raises(UserWarning):
            VilosunConfig.from_dict({**cfg, "something": 1})
    plain = {k: v for k, v in la[0]["mixer"].items() if k != "v_mix"}
    c = VilosunConfig.from_dict({**cfg, "layers": [{"type": "attention", "mixer": plain}]})
    assert c.first_values is None and model_class(cfg) is Vilosun


def test_weights_are_checked_against_the_configuration():
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    shapes = tensor_shapes(VilosunConfig.from_dict(cfg))
    assert {k: tuple(v.shape) for k, v in ts.items()} == shapes
    assert "l0.mix.vmix" not in shapes and shapes["l2.mix.vmix"] == () and "l1.norm2" not in shapes and shapes["bigram"] == (38, 45)
    for name in ("bigram", "l0.norm1b", "l0.rg1", "l0.rg1.b", "l0.rg2.b", "l0.norm2b", "l0.mix.q.b", "l0.mix.k.conv", "l0.mix.temp", "l0.mix.g",
                 "l1.mix.v.conv", "l1.mix.A_log", "l1.mix.dt_bias", "l1.mix.norm", "l1.mix.a", "l1.mix.g", "l0.mlp.router.b", "l0.mlp.e4.gate"):
        with pytest.raises(ValueError):
            Vilosun(cfg, {**ts, name: ts[name][:-1]}, **CPU)
    rnd = RandomTensors(cfg, 5)
    assert all(tuple(rnd[n].shape) == shapes[n] for n in rnd.keys())
    assert torch.equal(rnd["head"], RandomTensors(cfg, 5)["head"]) and float(rnd["l0.mix.q.b"].float().abs().max()) < 1
    eng = ServingEngine(build_model(cfg, 1, **CPU), num_pages=4, page_size=4, max_batch=1, max_context=16)
    assert len(eng.generate([[1, 2, 3]], 4)[0]) == 4


def test_folder_loads_through_the_registry(tmp_path):
    cfg, ts = H.CONFIGS["delta only"], H.tensors(H.CONFIGS["delta only"])
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    seq = H.prompts(cfg, [9])[0]
    eng = ServingEngine(load_model(str(tmp_path), **CPU), num_pages=8, page_size=4, max_batch=1, max_context=32)
    assert H.error(H.feed(eng, [seq], [[(0, 9)]])[0], H.expected(cfg, ts, [seq])[0]) < 1e-4


def test_cache_entries_of_several_parts():
    m = Vilosun(H.CONFIGS["odd"], H.tensors(H.CONFIGS["odd"]), **CPU)
    eng = ServingEngine(m, num_pages=3, page_size=4, max_batch=2, max_context=12)
    entries = eng.cache.entries
    assert len(entries) == 7 and [len(e) for e in entries[:6]] == [2, 2, 2, 2, 3, 2]
    pool, ring, first = entries[4]
    assert first is entries[2] and pool.shape == (3, 4, 2 * 8 + 2 * 16) and ring.shape == (2, 6, 6 * 7 + 2 * 7 + 2 * 13)
    state, ring = entries[1]
    assert state.shape == (2, 6, 10, 7) and state.dtype == torch.float32 and ring.shape == (2, 5, 2 * 30 + 42)
    assert entries[6].dtype == torch.int32 and entries[6].shape == (2, 1)
    specs = eng.backend.specs
    assert LayerCache.bytes_per_page(specs, 4, 2) == 4 * 2 * (2 * 16 + 2 * 16 + (2 * 16 + 2 * 16) + 48)
    assert LayerCache.bytes_per_slot(specs, 2) == sum(e.numel() * (2 if i == 1 else 4) for s in (1, 3, 5) for i, e in enumerate(entries[s])) // 2 \
        + sum(e[1].numel() * 2 for e in (entries[0], entries[2], entries[4])) // 2 + 4


# ----------------------------------------------------------------------------------------- mechanisms
def test_chunks_count_from_the_first_position():
    seen = lambda i, size: [j for j in range(i + 3) if O.visible(i, j, size)]
    assert seen(9, 5) == [5, 6, 7, 8, 9] and seen(10, 5) == [10] and seen(4, 5) == [0, 1, 2, 3, 4] and seen(6, 1) == [6] and seen(3, 99) == [0, 1, 2, 3]
    assert [O.slope(h, 4) for h in range(4)] == [0.25, 0.0625, 0.015625, 0.00390625] and O.slope(0, 3) == 2 ** (-8 / 3)


def test_group_norm_and_gated_step():
    x, w = 3 * randn(4, 12, seed=1), randn(12, seed=2)
    want = O.group_norm(x, w, 3, 1e-3)
    part = x[2, 4:8]
    assert torch.allclose(want[2, 4:8], part / math.sqrt(float((part * part).mean()) + 1e-3) * w[4:8])
    y, gate, post = randn(4, 12, seed=3), randn(4, 12, seed=4), randn(12, seed=5)
    after = x + O.group_norm(y * torch.sigmoid(gate), post, 3, 1e-3)
    pick = mo.group_step(x, 3, 1e-3, w, sub=mo.GatedOutput(y, gate, post), row_index=torch.tensor([3, 0]))
    assert torch.allclose(pick, O.group_norm(after, w, 3, 1e-3)[[3, 0]], atol=1e-6)
    h = mo.group_step(x, 3, 1e-3, w, sub=mo.GatedOutput(y, gate, post))
    assert torch.allclose(x, after, atol=1e-6) and torch.allclose(h, O.group_norm(after, w, 3, 1e-3), atol=1e-6)


def test_pairs_of_tokens_are_embedded():
    spec = {"buckets": 7, "mul_prev": 3, "mul_cur": 2}
    table, pairs = randn(9, 4, seed=1), randn(8, 4, seed=2)
    got = O.embed([5, 1, 8], table, 2.0, pairs, spec)
    assert torch.allclose(got, torch.stack([2 * table[5] + pairs[7], 2 * table[1] + pairs[(15 + 2) % 7], 2 * table[8] + pairs[(3 + 16) % 7]]))
    prev = torch.full((3, 1), 99, dtype=torch.int32)
    start, seqs, have = mo.EmbeddingStart(table, 2.0, pairs, 3, 2, prev), {0: [5, 1, 8, 0, 4], 2: [6, 6, 3]}, {0: 0, 2: 0}
    reqs = {s: Request(s, [], 0, pages=[s], slot=s) for s in seqs}
    for step in ([(0, 2)], [(0, 1), (2, 2)], [(2, 1), (0, 2)]):
        batch = StepBatch.build([(reqs[s], have[s], seqs[s][have[s]:have[s] + n]) for s, n in step], 8, 1, "cpu")
        x = torch.empty(batch.n_rows, 4)
        mo.group_step(x, 1, 1e-5, None, start=start, batch=batch)
        for r in range(batch.n_rows):
            s, p = step[batch.order[int(batch.row_seq[r])]][0], int(batch.positions[r])
            assert torch.allclose(x[r], O.embed(seqs[s], table, 2.0, pairs, spec)[p])
        for s, n in step:
            have[s] += n
    assert prev.reshape(-1).tolist() == [4, 99, 3]


def test_short_convolution():
    u, w = randn(6, 3, seed=1), randn(3, 4, seed=2)
    got = O.short_conv(u, w)
    assert torch.allclose(got[0], w[:, 3] * u[0]) and torch.allclose(got[4], w[:, 0] * u[1] + w[:, 1] * u[2] + w[:, 2] * u[3] + w[:, 3] * u[4])
    ring = torch.full((2, 4, 3), float("nan"))
    at = 0
    for n in (1, 2, 1, 1, 1):
        rows = mo.StepRows(torch.arange(at, at + n, dtype=torch.int32), torch.zeros(n, dtype=torch.int64), torch.tensor([1], dtype=torch.int32),
                           torch.zeros(n, dtype=torch.int32), 0, torch.tensor([0, n], dtype=torch.int32), [(0, n)])
        y = mo.short_conv(u[at:at + n], w.t().contiguous(), ring, rows, torch.empty(n, 3))
        assert torch.allclose(y, got[at:at + n], atol=1e-6)
        at += n
    assert torch.isnan(ring[0]).all() and torch.allclose(ring[1], u[[4, 5, 2, 3]])


def test_delta_rule_replaces_what_a_key_holds():
    """Without decay and with full strength a second write at the same key overwrites the first; an orthogonal key stays."""
    k = torch.eye(3, dtype=torch.float64)[[0, 1, 0, 1, 0]][:, None]
    v = randn(5, 1, 4, seed=1).double()
    one = torch.ones(5, 1, dtype=torch.float64)
    o = O.delta_rule(k, k, v, one, one)
    assert torch.allclose(o, v)
    beta = torch.tensor([1.0, 1.0, 0.0, 0.0, 0.25], dtype=torch.float64)[:, None]
    o = O.delta_rule(k, k, v, 0.5 * one, beta)
    assert torch.allclose(o[2], v[0] / 4) and torch.allclose(o[3], v[1] / 4) and torch.allclose(o[4], v[0] / 16 * 0.75 + v[4] / 4)


def test_routing_by_logit_with_a_bias():
    z, bias, slots = randn(40, 6, seed=1), randn(6, seed=2), torch.zeros(40, dtype=torch.int64)
    slots[7] = -1
    count = torch.zeros(6, dtype=torch.int32)
    choice, rank, weight = mo.moe_route(z, None, slots, 6, 2, count, bias=bias)
    want, share = O.route(z + bias, 2)
    live = slots >= 0
    assert torch.equal(choice[live], want[live].int()) and torch.allclose(weight[live], share[live], atol=1e-6) and (choice[7] == -1).all()


def _run(mixer, h, cache):
    """One prompt through a mixer: [tokens, width]."""
    pages = -(-len(h) // 4)
    req = Request(0, [0] * len(h), 0)
    req.pages, req.slot = list(range(pages)), 0
    return mixer(h, None, StepBatch.build([(req, 0, [0] * len(h))], 4, pages, "cpu"), cache)


def test_convolved_attention_options_combine():
    """A convolution with a sliding window, an element-wise gate and a sink; chunks with norms and rotation left out of the question."""
    heads, kv, dim, vdim, width, T = 4, 2, 6, 5, 9, 14
    ts = {"q": randn(heads * dim, width, seed=1), "k": randn(kv * dim, width, seed=2), "v": randn(kv * vdim, width, seed=3),
          "g": randn(heads * vdim, width, seed=4), "o": randn(width, heads * vdim, seed=5), "sink": randn(heads, seed=6)}
    ts.update({n + ".conv": randn(len(ts[n]), 3, seed=20 + i) for i, n in enumerate("qkv")})
    make = lambda **kw: GroupedAttention(ts.__getitem__, width, heads, kv, dim, vdim, 0.4, 4, 1e-4, torch.float32, "cpu", **kw)
    m = make(norm=None, conv=3, gated=True, sink=True, out_gate=(randn(width, width, seed=7), randn(width, seed=8)))
    h = randn(T, width, seed=11)
    got, gate = _run(m, h, (torch.zeros(4, 4, m.shape.cache_width), torch.zeros(1, 3, heads * dim + kv * (dim + vdim))))
    q, k, v = (O.short_conv(h @ ts[n].T, ts[n + ".conv"]).reshape(T, -1, d) for n, d in (("q", dim), ("k", dim), ("v", vdim)))
    out = []
    for n in range(heads):
        s = q[:, n] @ k[:, n // 2].T * 0.4
        for i in range(T):
            for j in range(T):
                if not 0 <= i - j < 4:
                    s[i, j] = -math.inf
        s = torch.softmax(torch.cat((s, ts["sink"][n].expand(T, 1)), 1), -1)[:, :-1]
        out.append(s @ v[:, n // 2])
    assert torch.allclose(got, (torch.cat(out, 1) * torch.sigmoid(h @ ts["g"].T)) @ ts["o"].T, atol=1e-4)
    assert torch.allclose(gate, h @ randn(width, width, seed=7).T + randn(width, seed=8), atol=1e-5)
    for kw in (dict(norm=None), dict(conv=3), dict(norm=None, conv=3, rot_dims=2), dict(norm=None, conv=3, kv_from=0), dict(temp=True), dict(mix_from=0),
               dict(norm=None, conv=3, chunked=True, keep=2), dict(norm=None, conv=3, slopes=[1.0] * 4, softcap=2.0)):
        with pytest.raises(ValueError):
            make(**kw)


def test_mixers_without_an_output_gate():
    ts = {"q": randn(6, 8, seed=1), "k": randn(6, 8, seed=2), "v": randn(20, 8, seed=3), "g": randn(20, 8, seed=4), "o": randn(8, 20, seed=5), "a": randn(4, 8, seed=6),
          "b": randn(4, 8, seed=7), "A_log": randn(4, seed=8), "dt_bias": randn(4, seed=9), "norm": 1 + randn(5, seed=10)}
    ts.update({n + ".conv": randn(len(ts[n]), 2, seed=20 + i) for i, n in enumerate("qkv")})
    m = DeltaRule(ts.__getitem__, 8, 4, 2, 3, 5, 2, 1e-4, torch.float32, "cpu")
    h = randn(9, 8, seed=11)
    got = _run(m, h, (torch.zeros(1, 4, 3, 5), torch.zeros(1, 2, 32)))
    assert torch.allclose(got, O.delta(h, ts.__getitem__, {"heads": 4, "kv_heads": 2, "dim": 3, "vdim": 5}, 1e-4), atol=1e-4)
    ts = {f"e{e}.{k}": randn(*((4, 8) if k != "down" else (8, 4)), seed=30 + 3 * e + i) for e in range(3) for i, k in enumerate(("gate", "up", "down"))}
    ts.update({"router": randn(3, 8, seed=50), "router.b": randn(3, seed=51)})
    m = RoutedExperts(ts.__getitem__, 8, 4, 3, 2, 0, None, torch.float32, "cpu", gated=True, choice="logits")
    x = torch.zeros(9, 8)
    mo.residual_norm(x, pending=m(h, torch.zeros(9, dtype=torch.int64), torch.zeros(3, dtype=torch.int32)))
    assert torch.allclose(x, O.mixture(h, ts.__getitem__, {"router": {"top": 2}}), atol=1e-4)


# --------------------------------------------------------------------------- model, cache, batches
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_whole_prompts_and_residuals_match_the_oracle(name):
    cfg = H.CONFIGS[name]
    ts = H.tensors(cfg)
    seqs = H.prompts(cfg, [1, 2, 29])
    eng = engine(cfg, ts)
    got = H.feed(eng, seqs, [[(0, 1)], [(1, 2), (2, 29)]])
    for g, w in zip(got, H.expected(cfg, ts, seqs)):
        assert H.error(g, w) < 2e-4
    req = eng.open("again")
    eng.sched.grow(req, 29)
    trace = []
    eng.backend.forward(StepBatch.build([(req, 0, seqs[2])], 4, eng.max_pages_per_req, eng.device), trace)
    want = O.Oracle(cfg, ts).residuals(seqs[2])
    assert len(trace) == want.shape[0]
    for a, b in zip(trace, want):
        assert float((a - b).abs().max()) < 2e-4 * max(1.0, float(b.abs().max()))


@pytest.mark.parametrize("name", ["odd", "tiles"])
def test_any_cut_and_any_company_gives_the_same_logits(name):
    cfg = H.CONFIGS[name]
    ts = H.tensors(cfg)
    seqs = H.prompts(cfg, [41, 7, 30, 2, 19])
    want = H.expected(cfg, ts, seqs)
    eng = engine(cfg, ts)
    for schedule in (sum([H.alone(i, len(s), [1]) for i, s in enumerate(seqs)], []),
                     sum([H.alone(i, len(s), [2, 3, 5]) for i, s in enumerate(seqs)], []),
                     sum([H.alone(i, len(s), [13, 1, 4]) for i, s in enumerate(seqs)], []),
                     H.mixed([len(s) for s in seqs], [[9, 1, 1, 2], [2], [1], [4, 7]])):
        for g, w in zip(H.feed(eng, seqs, schedule), want):
            assert H.error(g, w) < 2e-4
        assert eng.cache.allocator.free == eng.cache.num_pages and eng.cache.slot_allocator.free == 3 and not eng.sched.running


def _greedy(cfg, ts, prompt, n):
    o, ids = O.Oracle(cfg, ts, torch.float64), list(prompt)
    for _ in range(n):
        ids.append(int(o.logits(ids)[-1].argmax()))
    return ids[len(prompt):]


def test_greedy_generation_through_the_scheduler():
    """More requests than rows, prompts longer than a step's token budget, slots and pages that come round again."""
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    ps = H.prompts(cfg, [1, 23, 4, 30, 9])
    want = [_greedy(cfg, ts, p, 7) for p in ps]
    eng = engine(cfg, ts, max_prefill_tokens=8)
    assert eng.generate(ps, 7) == want
    assert eng.stats["prefill_steps"] > 5 and eng.stats["prefill_tokens"] == sum(map(len, ps))
    assert eng.cache.allocator.free == eng.cache.num_pages and eng.cache.slot_allocator.free == 3
    one = eng.backend.model.generate(torch.tensor(ps[3]), 7, temperature=0)
    assert one.reshape(-1).tolist() == want[3]
    torch.manual_seed(0)
    assert max(eng.generate(ps[:2], 5, temperature=0.7, top_k=3)[0]) < cfg["vocab"]


def test_logits_do_not_depend_on_what_else_is_live():
    """A request that sits out steps while others come, go and take over their pages and slots."""
    cfg = H.CONFIGS["tiles"]
    ts = H.tensors(cfg, 3)
    a, b, c = H.prompts(cfg, [22, 15, 17], seed=4)
    eng = engine(cfg, ts, num_pages=12)
    schedule = [[(0, 6)], [(1, 15)], [(0, 1), (2, 9)], [(2, 2)], [(2, 1)], [(0, 3), (2, 5)], [(0, 12)]]
    for g, w in zip(H.feed(eng, [a, b, c], schedule), H.expected(cfg, ts, [a, b, c])):
        assert H.error(g, w) < 2e-4


def test_cancel_during_a_long_prompt_frees_everything():
    cfg = H.CONFIGS["tiles"]
    eng = engine(cfg, H.tensors(cfg), max_prefill_tokens=5)
    eng._realtime, eng._virtual = False, float("inf")
    r = Request(0, H.prompts(cfg, [40])[0], 4)
    eng.sched.add(r)
    eng.step(float("inf"))
    assert r.fed == 5 and eng.cancel(r)
    assert eng.cache.allocator.free == eng.cache.num_pages and eng.cache.slot_allocator.free == 3 and eng.sched.idle


# -------------------------------------------------------------------------------------- command lines
def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from llm_systems_from_scratch_b200.serving import trace
    cfg, ts = H.CONFIGS["odd"], H.tensors(H.CONFIGS["odd"])
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    a, b = H.prompts(cfg, [12, 5])
    wa = H.expected(cfg, ts, [a])[0]
    eng = trace.open_engine(str(tmp_path), torch.float32, 128, "cpu")
    said = []
    lines = [json.dumps(s) for s in (
        {"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [6, 0]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[7:8], "want": []}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[8:], "want": [3]}], "end": ["a"]})]
    trace.replay(eng, lines, str(tmp_path), lambda text, flush: said.append(text))
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    read = lambda n, rows: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(rows, cfg["vocab"])
    assert H.error(read(0, 2), wa[[6, 0]]) < 2e-4 and H.error(read(2, 1), wa[[11]]) < 2e-4


def test_generate_and_serve_commands(tmp_path, capsys):
    import generate
    import serve
    cfg, ts = H.CONFIGS["odd"], H.tensors(H.CONFIGS["odd"])
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    prompt = H.prompts(cfg, [6])[0]
    generate.main(["--model", str(tmp_path), "--dtype", "float32", "--device", "cpu", "--temperature", "0", "--max-tokens", "5",
                   "--prompt-ids", ",".join(map(str, prompt))])
    assert capsys.readouterr().out.strip() == ",".join(map(str, _greedy(cfg, ts, prompt, 5)))
    if torch.cuda.is_available():
        return
    (tmp_path / "s.yaml").write_text(json.dumps({"model": cfg, "serving": {
        "max_batch": 3, "max_context": 48, "num_requests": 5, "prompt_len": [2, 20], "output_len": [2, 6], "page_size": 4}}))
    serve.main(["--config", str(tmp_path / "s.yaml"), "--offline"])
    rec = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert rec["requests"] == 5 and rec["model"] == "Vilosun" and rec["output_tokens"] > 0


def test_serving_configuration_and_kernel_sources():
    import os
    from llm_systems_from_scratch_b200 import build_ext
    from llm_systems_from_scratch_b200.utils.config import load_config, validate
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = validate(load_config(os.path.join(root, "configures", "serve_vilosun.yaml")), require_dataset=False)
    layers = VilosunConfig.from_dict(cfg["model"]).layers
    assert len(layers) == 24 and {la.type for la in layers} == {"delta", "attention"}
    assert set(Vilosun.KERNELS) <= build_ext.MIXERS <= {s.name for s in build_ext.sources()}
