"""Genedra on the CPU statements of its kernels: configuration, weights, scheduling, caches and batches against the plain
oracle (the kernels themselves: tests/test_gpu_genedra.py)."""
import json
import math
import warnings

import pytest
import torch

import genedra_helpers as H
import genedra_oracle as O
from llm_systems_from_scratch_b200.models.genedra import Genedra, GenedraConfig, RandomTensors, tensor_shapes
from llm_systems_from_scratch_b200.models.mixers import GroupedAttention, LatentAttention, RotaryTable
from llm_systems_from_scratch_b200.models.registry import build_model, load_model, model_class
from llm_systems_from_scratch_b200.ops import mixer_ops as mo
from llm_systems_from_scratch_b200.serving import Request, ServingEngine
from llm_systems_from_scratch_b200.serving.batch import StepBatch
from llm_systems_from_scratch_b200.serving.kv_cache import LayerCache
from llm_systems_from_scratch_b200.utils import safetensors as st

CPU = dict(dtype=torch.float32, device="cpu")


def engine(cfg, ts, **kw):
    args = dict(num_pages=24, page_size=4, max_batch=3, max_context=96)
    args.update(kw)
    return ServingEngine(Genedra(cfg, ts, **CPU), **args)


def randn(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed))


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_is_read_and_checked():
    cfg = H.CONFIGS["odd"]
    c = GenedraConfig.from_dict(cfg)
    assert [la.type for la in c.layers].count("attention") == 2 and c.layers[2].mixer["kv_from"] == 1 and c.layers[4].mixer["kv_from"] is None
    assert (c.eps, c.embed_scale, c.gain, c.logit_softcap) == (1e-4, 1.0, 1.0, 7.0) and c.layers[3].mlp is None
    la = cfg["layers"]
    mix = lambda i, **kw: {**la[i], "mixer": {**la[i]["mixer"], **kw}}
    mlp = lambda i, **kw: {**la[i], "mlp": {**la[i]["mlp"], **kw}}
    bad = ([{**la[0], "type": "convolution"}], [mix(0, kv_heads=4)], [mix(0, mask={"size": 0, "keep_first": 2})], [mix(0, softcap=0.0)],
           [mix(0, mask={"size": 3, "keep_first": -1})], [mix(1, rot_dim=8)], [la[2]], [la[0], mix(2, kv_from=0)], [*la[:3], mix(2, kv_from=2)],
           [*la[:2], mix(2, kv_rank=20)], [*la[:2], mix(2, rot={"base": 7.0, "dims": 6})], [mlp(0, kind="sparse")],
           [mlp(0, router={"experts": 5, "top": 8, "identity": 2})], [mlp(0, expert={})], [{"type": "attention", "mixer": {"heads": 2}}])
    for layers in bad:
        with pytest.raises(ValueError):
            GenedraConfig.from_dict({**cfg, "layers": layers})
    for key in ("embedding", "residual_mult", "logit_softcap"):
        with pytest.raises(ValueError):
            GenedraConfig.from_dict({k: v for k, v in cfg.items() if k != key})
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        with pytest.raises(UserWarning):
            GenedraConfig.from_dict({**cfg, "something": 1})
    plain = mix(0, mask={"size": 4}, rot={"base": 100.0, "dims": 4})
    m = GenedraConfig.from_dict({**cfg, "layers": [plain]}).layers[0].mixer
    assert m["rot"]["scaling"] is None and m["mask"]["keep_first"] == 0 and model_class(cfg) is Genedra


def test_weights_are_checked_against_the_configuration():
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    shapes = tensor_shapes(GenedraConfig.from_dict(cfg))
    assert {k: tuple(v.shape) for k, v in ts.items()} == shapes
    assert "l2.mix.dkv" not in shapes and "l3.norm2" not in shapes and "l0.mlp.e5.up" not in shapes and shapes["l0.mlp.router"] == (7, 44)
    for name in ("l1.mix.dkv", "l1.mix.dkv.norm", "l0.mix.q.b", "l0.mix.q.norm", "l0.mix.sink", "l0.mix.o.b", "l0.norm1", "l0.mlp.correction",
                 "l0.mlp.e4.up", "l0.mlp.shared.sg", "l1.mlp.down", "l5.mix.g", "l2.mix.uk"):
        with pytest.raises(ValueError):
            Genedra(cfg, {**ts, name: ts[name][:-1]}, **CPU)
    rnd = RandomTensors(cfg, 5)
    assert all(tuple(rnd[n].shape) == shapes[n] for n in rnd.keys())
    assert torch.equal(rnd["head"], RandomTensors(cfg, 5)["head"]) and float(rnd["final.norm"].float().abs().max()) < 1
    eng = ServingEngine(build_model(cfg, 1, **CPU), num_pages=4, page_size=4, max_batch=1, max_context=16)
    assert len(eng.generate([[1, 2, 3]], 4)[0]) == 4


def test_folder_loads_through_the_registry(tmp_path):
    cfg, ts = H.CONFIGS["latent only"], H.tensors(H.CONFIGS["latent only"])
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    seq = H.prompts(cfg, [9])[0]
    eng = ServingEngine(load_model(str(tmp_path), **CPU), num_pages=8, page_size=4, max_batch=1, max_context=32)
    assert H.error(H.feed(eng, [seq], [[(0, 9)]])[0], H.expected(cfg, ts, [seq])[0]) < 1e-4


def test_a_shared_layer_has_no_pool_of_its_own():
    m = Genedra(H.CONFIGS["odd"], H.tensors(H.CONFIGS["odd"]), **CPU)
    specs = [layer.mixer.cache_spec() for layer in m.runs]
    assert [type(s).__name__ for s in specs] == ["PagedSpec", "PagedSpec", "SharedSpec", "PagedSpec", "PagedSpec", "SharedSpec"]
    cache = LayerCache(specs, 3, 4, 2, "cpu", torch.float32)
    assert cache.entries[2] is cache.entries[1] and cache.entries[5] is cache.entries[1]
    assert specs[1].width == 24 + 8                          # latent and rotated part, each in whole pieces of eight


# ----------------------------------------------------------------------------------------- mechanisms
def test_rotation_layouts_and_linear_scaling():
    pos = torch.tensor([0, 1, 777, 100000])
    for rot in ({"base": 900.0, "dims": 6}, {"base": 1e6, "dims": 10, "scaling": {"factor": 3.0}}, {"base": 50.0, "dims": 2, "scaling": None}):
        table = RotaryTable(rot["base"], rot["dims"], "cpu", rot.get("scaling"))
        table.resize(100001)
        x = torch.randn(4, 2, 12, dtype=torch.float64)
        inter, half = O.rotate_interleaved(x, pos, rot), O.rotate_half(x, pos, rot)
        h = rot["dims"] // 2
        for p in range(4):
            for i, f in enumerate(O.frequencies(rot)):
                assert f == rot["base"] ** (-2 * i / rot["dims"]) / (3.0 if rot.get("scaling") else 1.0)
                c, s = math.cos(int(pos[p]) * f), math.sin(int(pos[p]) * f)
                assert abs(float(table.table[0, pos[p], i]) - c) < 1e-6 and abs(float(table.table[1, pos[p], i]) - s) < 1e-6
                u, v = x[p, 0, 2 * i], x[p, 0, 2 * i + 1]
                assert abs(float(inter[p, 0, 2 * i + 1] - (v * c + u * s))) < 1e-9
                u, v = x[p, 1, i], x[p, 1, i + h]
                assert abs(float(half[p, 1, i] - (u * c - v * s))) < 1e-9
        assert torch.equal(inter[..., rot["dims"]:], x[..., rot["dims"]:]) and torch.equal(half[..., rot["dims"]:], x[..., rot["dims"]:])


def test_window_beside_kept_tokens():
    seen = lambda i, size, keep: [j for j in range(i + 3) if O.visible(i, j, size, keep)]
    assert seen(9, 3, 2) == [0, 1, 7, 8, 9] and seen(3, 3, 2) == [0, 1, 2, 3] and seen(0, 1, 5) == [0] and seen(6, 1, 0) == [6]
    assert seen(5, 100, 2) == list(range(6)) and seen(5, 2, 100) == list(range(6))


def test_sink_takes_its_share():
    """One key: the output is the value times exp(s) / (exp(s) + exp(sink)), s capped."""
    q, k, v = randn(1, 2, 3, seed=1).double(), randn(1, 1, 3, seed=2).double(), randn(1, 1, 4, seed=3).double()
    sink = torch.tensor([0.3, -2.0], dtype=torch.float64)
    got = O.sink_attention(q, k, v, 0.7, 1.5, 4, 0, sink)
    for h in range(2):
        s = 1.5 * math.tanh(0.7 * float(q[0, h] @ k[0, 0]) / 1.5)
        assert torch.allclose(got[0, h], v[0, 0] * math.exp(s) / (math.exp(s) + math.exp(float(sink[h]))))


def test_finished_products():
    a, w, b, c = randn(4, 6, seed=1), randn(5, 6, seed=2), randn(5, seed=3), randn(4, 5, seed=4)
    r = a @ w.t()
    assert torch.allclose(mo.linear(a, w, bias=b), r + b, atol=1e-6)
    assert torch.allclose(mo.linear(a, w, act="gelu"), O.gelu(r), atol=1e-6)
    assert torch.allclose(mo.linear(a, w, act="cap", cap=1.3), O.softcap(r, 1.3), atol=1e-6)
    out = c.clone()
    mo.linear(a, w, out=out, accumulate=True, alpha=0.3, bias=b)
    assert torch.allclose(out, c + 0.3 * (r + b), atol=1e-6)


def test_routing_and_dispatch():
    rows, experts, identity, top = 300, 5, 2, 3
    z, corr, slots = 2 * randn(rows, experts + identity, seed=1), 0.1 * randn(experts + identity, seed=2), torch.zeros(rows, dtype=torch.int64)
    slots[::9] = -1
    count = torch.zeros(experts, dtype=torch.int32)
    choice, rank, weight = mo.moe_route(z, corr, slots, experts, top, count)
    want, wweight = O.route(z, torch.eye(experts + identity), corr, top)
    live = slots >= 0
    assert torch.equal(choice[live].sort(-1).values, want[live].int().sort(-1).values) and (choice[~live] == -1).all()
    dense = lambda c, w: torch.zeros(len(c), experts + identity).scatter(1, c.long(), w)
    assert torch.allclose(dense(choice[live], weight[live]), dense(want[live], wweight[live]), atol=1e-6)
    assert torch.allclose(weight[live].sum(1), torch.ones(int(live.sum())))
    assert int(count.sum()) == int((choice[live] < experts).sum())
    h = randn(rows, 6, seed=3)
    xg, pos, group = mo.moe_dispatch(h, choice, rank, count)
    for e in range(experts):
        used = pos[choice == e]
        assert used.unique().numel() == used.numel() == int(count[e]) and (group[(used // mo.TILE).long()] == e).all()
    assert (pos[choice >= experts] == -2).all() and (pos[~live] == -1).all()
    r, k = ((choice >= 0) & (choice < experts)).nonzero(as_tuple=True)
    assert torch.equal(xg[pos[r, k].long()], h[r])
    # two more experts that every row uses, weighted by one more logit
    z2 = torch.cat((z, randn(rows, 1, seed=4)), 1)
    choice, rank, weight = mo.moe_route(z2, corr, slots, experts, top, count.zero_(), 2)
    assert torch.allclose(weight[live, top:], torch.sigmoid(z2[live, -1:]).expand(-1, 2)) and float(weight[~live].abs().sum()) == 0.0
    xg, more, group = mo.moe_dispatch(h, choice, rank, count, 2)
    assert torch.equal(more[:, :top], pos) and (more[~live] == -1).all()
    for a in range(2):
        assert (group[(more[live, top + a] // mo.TILE).long()] == experts + a).all() and torch.equal(xg[more[live, top + a].long()], h[live])


def test_expert_outputs_join_the_residual_stream():
    x, z, s, w = randn(3, 5, seed=1), randn(3, 5, seed=2), randn(3, 5, seed=3), randn(5, seed=4)
    y, pos = randn(4, 5, seed=5), torch.tensor([[2, -2], [0, 3], [-1, -1]], dtype=torch.int32)
    weight, gate = torch.rand(3, 2), randn(3, 2, seed=6)
    want = x + 0.4 * (torch.stack([weight[0, 0] * y[2] + weight[0, 1] * z[0], weight[1, 0] * y[0] + weight[1, 1] * y[3], torch.zeros(5)])
                      + torch.sigmoid(gate[:, 1:]) * s)
    ex = mo.ExpertOutputs(y, pos, 0.4, weight, z, s, gate[:, 1])
    h, _ = mo.residual_norm(x.clone(), w, 1e-3, row_index=torch.tensor([2, 0]), pending=ex, w_offset=1.0)
    assert torch.allclose(h, O.centred_norm(want, w, 1e-3)[[2, 0]], atol=1e-6)
    h, _ = mo.residual_norm(x, w, 1e-3, pending=ex, w_offset=1.0)
    assert torch.allclose(x, want, atol=1e-6) and torch.allclose(h, O.centred_norm(want, w, 1e-3), atol=1e-6)
    emb = randn(7, 5, seed=7)
    mo.residual_norm(x, tokens=torch.tensor([6, 0, 6]), embed=emb, embed_scale=2.5)
    assert torch.allclose(x, 2.5 * emb[[6, 0, 6]])


def _run_mixer(mixer, h, cache):
    """One prompt through a mixer: [tokens, width]."""
    req = Request(0, [0] * len(h), 0)
    req.pages, req.slot = list(range(cache.shape[0])), 0
    batch = StepBatch.build([(req, 0, [0] * len(h))], cache.shape[1], cache.shape[0], "cpu")
    x = torch.zeros_like(h)
    mixer(h, x, batch, cache)
    return x


def test_latent_attention_with_a_low_rank_query_and_rotation():
    """Options that no single model combines: W_q in two factors beside rotated parts, element-wise gate, a window."""
    heads, dim, vdim, qr, kvr, rd, width, T = 3, 5, 6, 7, 9, 4, 10, 12
    ts = {"dq": randn(qr, width, seed=1), "dq.norm": 1 + 0.1 * randn(qr, seed=2), "uq": randn(heads * (dim + rd), qr, seed=3),
          "dkv": randn(kvr + rd, width, seed=4), "dkv.norm": 1 + 0.1 * randn(kvr, seed=5), "uk": randn(heads * dim, kvr, seed=6),
          "uv": randn(heads * vdim, kvr, seed=7), "g": randn(heads * vdim, width, seed=8), "o": randn(width, heads * vdim, seed=9)}
    rope = RotaryTable(30.0, rd, "cpu")
    rope.resize(T)
    m = LatentAttention(ts.__getitem__, width, heads, dim, vdim, qr, kvr, 0.3, 5, 1e-4, torch.float32, "cpu", rot_dim=rd, rope=rope)
    h = randn(T, width, seed=10)
    got = _run_mixer(m, h, torch.zeros(4, 4, m.cached))
    spec = {"kv_rank": kvr, "rot": {"base": 30.0, "dims": rd}}
    c, kr = O.latent_keys(h, ts.__getitem__, spec, 1e-4)
    q = (O.rms_norm(h @ ts["dq"].T, ts["dq.norm"], 1e-4) @ ts["uq"].T).reshape(T, heads, dim + rd)
    qr_ = O.rotate_interleaved(q[..., dim:], torch.arange(T), spec["rot"])
    i = torch.arange(T)
    hidden = (i[:, None] < i[None]) | (i[:, None] - i[None] >= 5)
    out = []
    for n in range(heads):
        k = c @ ts["uk"][n * dim:(n + 1) * dim].T
        s = (q[:, n, :dim] @ k.T + qr_[:, n] @ kr.T) * 0.3
        out.append(torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ (c @ ts["uv"][n * vdim:(n + 1) * vdim].T))
    want = (torch.cat(out, 1) * torch.sigmoid(h @ ts["g"].T)) @ ts["o"].T
    assert torch.allclose(got, want, atol=1e-4)


def test_grouped_attention_options_combine():
    """A distance bias and a gate beside caps, kept tokens and biases."""
    heads, kv, dim, vdim, width, T = 4, 2, 6, 5, 9, 14
    ts = {"q": randn(heads * dim, width, seed=1), "k": randn(kv * dim, width, seed=2), "v": randn(kv * vdim, width, seed=3),
          "g": randn(heads * vdim, width, seed=4), "o": randn(width, heads * vdim, seed=5), "q.norm": 1 + randn(dim, seed=6),
          "k.norm": 1 + randn(dim, seed=7), "rel": randn(6, heads, seed=8), "o.b": randn(width, seed=9)}
    ts.update({n + ".b": randn(len(ts[n]), seed=20 + i) for i, n in enumerate("qkv")})
    m = GroupedAttention(ts.__getitem__, width, heads, kv, dim, vdim, 0.4, 4, 1e-4, torch.float32, "cpu", bias_max=10, gated=True, keep=3,
                         softcap=1.2, biased=True, gain=0.5)
    h = randn(T, width, seed=11)
    got = _run_mixer(m, h, torch.zeros(4, 4, m.shape.cache_width))
    proj = lambda n: h @ ts[n].T + ts[n + ".b"]
    q, k = (O.rms_norm(proj(n).reshape(T, -1, dim), ts[n + ".norm"], 1e-4) for n in "qk")
    v, out, table = proj("v").reshape(T, kv, vdim), [], m.shape.bias
    for n in range(heads):
        s = O.softcap(q[:, n] @ k[:, n // 2].T * 0.4, 1.2)
        for i in range(T):
            for j in range(T):
                s[i, j] = s[i, j] + table[n, min(i - j, table.shape[1] - 1)] if O.visible(i, j, 4, 3) else -math.inf
        out.append(torch.softmax(s, -1) @ v[:, n // 2])
    want = 0.5 * ((torch.cat(out, 1) * torch.sigmoid(h @ ts["g"].T)) @ ts["o"].T + ts["o.b"])
    assert torch.allclose(got, want, atol=1e-4)
    for kw in (dict(difference=0.1, sink=True), dict(difference=0.1, norm="projection"), dict(norm="row")):
        with pytest.raises(ValueError):
            GroupedAttention(ts.__getitem__, width, heads, kv, dim, vdim, 0.4, 4, 1e-4, torch.float32, "cpu", **kw)


# --------------------------------------------------------------------------- model, cache, batches
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_whole_prompts_and_residuals_match_the_oracle(name):
    cfg = H.CONFIGS[name]
    ts = H.tensors(cfg)
    seqs = H.prompts(cfg, [1, 2, 29])
    eng = engine(cfg, ts)
    got = H.feed(eng, seqs, [[(0, 1)], [(1, 2), (2, 29)]], poison=True)
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
        for g, w in zip(H.feed(eng, seqs, schedule, poison=True), want):
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
    """A request that sits out steps while others come, go and take over their pages."""
    cfg = H.CONFIGS["tiles"]
    ts = H.tensors(cfg, 3)
    a, b, c = H.prompts(cfg, [22, 15, 17], seed=4)
    eng = engine(cfg, ts, num_pages=12)
    schedule = [[(0, 6)], [(1, 15)], [(0, 1), (2, 9)], [(2, 2)], [(2, 1)], [(0, 3), (2, 5)], [(0, 12)]]
    for g, w in zip(H.feed(eng, [a, b, c], schedule, poison=True), H.expected(cfg, ts, [a, b, c])):
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
    assert rec["requests"] == 5 and rec["model"] == "Genedra" and rec["output_tokens"] > 0


def test_serving_configuration_and_kernel_sources():
    import os
    from llm_systems_from_scratch_b200 import build_ext
    from llm_systems_from_scratch_b200.utils.config import load_config, validate
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = validate(load_config(os.path.join(root, "configures", "serve_genedra.yaml")), require_dataset=False)
    layers = GenedraConfig.from_dict(cfg["model"]).layers
    assert len(layers) == 24 and {la.type for la in layers} == {"latent_attention", "attention"}
    assert set(Genedra.KERNELS) <= build_ext.MIXERS <= {s.name for s in build_ext.sources()}
