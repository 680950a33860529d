"""Tedirax on the CPU statements of its kernels: configuration, weights, scheduling, caches and batches against the plain
oracle (the kernels themselves: tests/test_gpu_tedirax.py)."""
import json

import pytest
import torch

import tedirax_helpers as H
import tedirax_oracle as O
from llm_systems_from_scratch_b200.models.registry import build_model, load_model, model_class
from llm_systems_from_scratch_b200.models.tedirax import RandomTensors, Tedirax, TediraxConfig, tensor_shapes
from llm_systems_from_scratch_b200.ops import mixer_ops as mo
from llm_systems_from_scratch_b200.serving import Request, ServingEngine
from llm_systems_from_scratch_b200.utils import safetensors as st

CPU = dict(dtype=torch.float32, device="cpu")


def engine(cfg, ts, **kw):
    args = dict(num_pages=24, page_size=4, max_batch=3, max_context=96)
    args.update(kw)
    return ServingEngine(Tedirax(cfg, ts, **CPU), **args)


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_is_read_and_checked():
    cfg = H.CONFIGS["odd"]
    c = TediraxConfig.from_dict(cfg)
    assert c.runs() == [0, 1, 2, 1, 2] and O.layer_order(cfg) == c.runs() and c.eps == 1e-4
    assert TediraxConfig.from_dict({**cfg, "loop": None}).runs() == [0, 1, 2]
    assert TediraxConfig.from_dict({k: v for k, v in cfg.items() if k != "loop"}).runs() == [0, 1, 2]
    for change in ({"layers": [{**cfg["layers"][0], "type": "convolution"}]}, {"width": None, "layers": [{"type": "retention"}]},
                   {"loop": {"start": 2, "stop": 9, "times": 1}},
                   {"layers": [{**cfg["layers"][0], "mlp": {**H.moe(4, 2, 1), "kind": "dense"}}]}):
        with pytest.raises((ValueError, TypeError)):
            TediraxConfig.from_dict({**cfg, **change})
    assert model_class(cfg) is Tedirax and model_class({"vocab_size": 5}).__name__ == "TransformerLM"
    with pytest.raises(ValueError):
        model_class({"architecture": "Nothing"})


def test_weights_are_checked_against_the_configuration():
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    assert {k: tuple(v.shape) for k, v in ts.items()} == tensor_shapes(TediraxConfig.from_dict(cfg))
    bad = dict(ts)
    bad["l1.mix.uk"] = ts["l1.mix.uk"][:-1]
    with pytest.raises(ValueError):
        Tedirax(cfg, bad, **CPU)
    bad = dict(ts)
    bad["l0.mlp.table"] = ts["l0.mlp.table"] + 3
    with pytest.raises(ValueError):
        Tedirax(cfg, bad, **CPU)
    rnd = RandomTensors(cfg, 5)
    for name in rnd.keys():
        assert tuple(rnd[name].shape) == tuple(ts[name].shape)
    assert torch.equal(rnd["head"], RandomTensors(cfg, 5)["head"])


def test_safetensors_round_trip_and_damage(tmp_path):
    path = str(tmp_path / "x.safetensors")
    ts = {"a": torch.randn(3, 5).bfloat16(), "t": torch.arange(6, dtype=torch.int32).view(2, 3), "s": torch.randn(4), "e": torch.empty(0, 2)}
    st.save(path, ts)
    f = st.SafetensorsFile(path)
    assert set(f.keys()) == set(ts) and f.shape("a") == (3, 5) and all(torch.equal(f[k], v) for k, v in ts.items())
    with pytest.raises(KeyError):
        f["b"]
    raw = open(path, "rb").read()
    open(path, "wb").write(raw[:-8])
    with pytest.raises(ValueError):
        st.SafetensorsFile(path)


def test_folder_loads_through_the_registry(tmp_path):
    cfg, ts = H.CONFIGS["latent only"], H.tensors(H.CONFIGS["latent only"])
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    model = load_model(str(tmp_path), **CPU)
    seq = H.prompts(cfg, [9])[0]
    eng = ServingEngine(model, num_pages=8, page_size=4, max_batch=1, max_context=32)
    assert H.error(H.feed(eng, [seq], [[(0, 9)]])[0], H.expected(cfg, ts, [seq])[0]) < 1e-4


# ----------------------------------------------------------------------------------------- mechanisms
def test_rotation_leaves_the_other_dimensions_and_uses_double_angles():
    x = torch.randn(5, 2, 10, dtype=torch.float64)
    pos = torch.tensor([0, 1, 7, 3000, 100000])
    y = O.rotate_half(x, pos, 1000.0, 6)
    assert torch.equal(y[..., 6:], x[..., 6:]) and torch.allclose(y[0], x[0])
    f = 1000.0 ** (-2 * 1 / 6)
    a = torch.tensor(100000 * f, dtype=torch.float64)
    assert torch.allclose(y[4, 0, 1], x[4, 0, 1] * a.cos() - x[4, 0, 4] * a.sin())
    assert torch.allclose(y[4, 0, 4], x[4, 0, 4] * a.cos() + x[4, 0, 1] * a.sin())


def test_residual_norm_statement():
    g = torch.Generator().manual_seed(0)
    emb, w = torch.randn(11, 7, generator=g), torch.randn(7, generator=g)
    tok = torch.tensor([3, 3, 10, 0])
    x = torch.empty(4, 7)
    pos = torch.tensor([[2, 0], [1, -1], [-1, -1], [3, 4]], dtype=torch.int32)
    y = torch.randn(5, 7, generator=g)
    h, xg = mo.residual_norm(x, w, 1e-3, tokens=tok, embed=emb, scatter=(pos, 6))
    assert torch.equal(x, emb[tok]) and torch.allclose(h, O.rms_norm(emb[tok], w, 1e-3), atol=1e-6)
    assert torch.equal(xg[2], h[0]) and torch.equal(xg[0], h[0]) and torch.equal(xg[1], h[1]) and torch.equal(xg[4], h[3])
    want = x + 0.5 * torch.stack([y[2] + y[0], y[1], torch.zeros(7), y[3] + y[4]])
    keep = x.clone()
    h2, _ = mo.residual_norm(x, w, 1e-3, row_index=torch.tensor([3, 1]), pending=(y, pos, 0.5))
    assert torch.equal(x, keep) and torch.allclose(h2, O.rms_norm(want, w, 1e-3)[[3, 1]], atol=1e-6)
    mo.residual_norm(x, pending=(y, pos, 0.5))
    assert torch.allclose(x, want, atol=1e-6)


def test_expert_plan_sorts_rows_into_tiles():
    g = torch.Generator().manual_seed(0)
    table = torch.stack([torch.randperm(5, generator=g)[:3] for _ in range(40)]).int()
    tokens, slots = torch.randint(0, 40, (200,), generator=g), torch.zeros(200, dtype=torch.int64)
    slots[::7] = -1
    (pos,), (group,) = mo.moe_plan(tokens, slots, [table], [5])
    assert group.numel() == mo.plan_tiles(200, 5, 3) and (pos[slots < 0] == -1).all()
    used = pos[slots >= 0]
    assert used.unique().numel() == used.numel()
    assert torch.equal(group[(used // mo.TILE).long()], table[tokens[slots >= 0]])
    # the bound is never exceeded: all rows on one expert, one row alone, every expert one row
    for rows, n, top in ((1, 5, 3), (128, 5, 1), (129, 2, 2), (700, 300, 7)):
        t = torch.arange(top).int().repeat(9, 1) if n < 20 else torch.stack([torch.randperm(n, generator=g)[:top] for _ in range(9)]).int()
        p, gr = mo.moe_plan(torch.randint(0, 9, (rows,), generator=g), torch.zeros(rows, dtype=torch.int64), [t], [n])
        assert int(p[0].max()) < mo.plan_tiles(rows, n, top) * mo.TILE and int((gr[0] >= 0).sum()) <= mo.plan_tiles(rows, n, top)


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
    from llm_systems_from_scratch_b200.serving.batch import StepBatch
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
    stop = want[1][2]
    assert eng.generate([ps[1]], 7, eos_token_id=stop)[0] == want[1][:want[1].index(stop) + 1]
    one = eng.backend.model.generate(torch.tensor(ps[3]), 7, temperature=0)
    assert one.reshape(-1).tolist() == want[3]
    torch.manual_seed(0)
    assert max(eng.generate(ps[:2], 5, temperature=0.7, top_k=3)[0]) < cfg["vocab"]


def test_cancel_during_a_long_prompt_frees_everything():
    cfg = H.CONFIGS["retention only"]
    eng = engine(cfg, H.tensors(cfg), max_prefill_tokens=5)
    eng._realtime, eng._virtual = False, float("inf")
    r = Request(0, H.prompts(cfg, [40])[0], 4)
    eng.sched.add(r)
    eng.step(float("inf"))
    assert r.fed == 5 and eng.cancel(r) and not eng.cancel(r)
    assert eng.cache.allocator.free == eng.cache.num_pages and eng.cache.slot_allocator.free == 3 and eng.sched.idle


def test_limits_are_refused():
    cfg = H.CONFIGS["latent only"]
    eng = engine(cfg, H.tensors(cfg), num_pages=2)
    rs = [eng.open(i) for i in range(3)]
    with pytest.raises(MemoryError):
        eng.open(3)
    with pytest.raises(MemoryError):
        eng.extend([(rs[0], [1] * 9, [])])
    with pytest.raises(ValueError):
        eng.extend([(rs[1], [], [])])
    with pytest.raises(ValueError):
        eng.extend([(rs[1], [1, 2], [2])])


def test_transformer_runs_portions_beside_single_tokens():
    """The same step function on the TransformerLM: portions that continue a prompt read their earlier keys from the pages."""
    cfg = dict(vocab_size=61, context_length=64, d_model=32, num_layers=2, num_heads=2, d_ff=64, rope_theta=10000.0)
    model = build_model(cfg, seed=1, device="cpu")
    seqs = H.prompts({"vocab": 61}, [20, 5, 13])
    want = [model(torch.tensor([s]))[0] for s in seqs]
    eng = ServingEngine(model, num_pages=16, page_size=4, max_batch=3, max_context=64)
    for g, w in zip(H.feed(eng, seqs, H.mixed([20, 5, 13], [[7, 1, 1], [2], [3, 1]])), want):
        assert H.error(g, w.detach()) < 1e-4


# -------------------------------------------------------------------------------------- command lines
def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from llm_systems_from_scratch_b200.serving import trace
    cfg, ts = H.CONFIGS["odd"], H.tensors(H.CONFIGS["odd"])
    folder = tmp_path / "m"
    folder.mkdir()
    st.save(str(folder / "model.safetensors"), ts)
    (folder / "config.json").write_text(json.dumps(cfg))
    a, b = H.prompts(cfg, [12, 5])
    wa, wb = H.expected(cfg, ts, [a, b])
    eng = trace.open_engine(str(folder), torch.float32, 128, "cpu")
    said = []
    lines = [json.dumps(s) for s in (
        {"step": 0, "entries": [{"id": "a", "tokens": a[:7], "want": [6, 0]}], "end": []},
        {"step": 1, "entries": [{"id": "b", "tokens": b, "want": []}, {"id": "a", "tokens": a[7:8], "want": []}], "end": ["b"]},
        {"step": 2, "entries": [{"id": "a", "tokens": a[8:], "want": [3]}], "end": ["a"]})]
    trace.replay(eng, lines, str(tmp_path), lambda text, flush: said.append(text))
    assert said == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    read = lambda n, rows: torch.frombuffer(bytearray((tmp_path / f"{n}.f32").read_bytes()), dtype=torch.float32).view(rows, cfg["vocab"])
    assert H.error(read(0, 2), wa[[6, 0]]) < 2e-4 and H.error(read(2, 1), wa[[11]]) < 2e-4 and wb.shape[0] == 5


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
    assert rec["requests"] == 5 and rec["model"] == "Tedirax" and rec["output_tokens"] > 0
