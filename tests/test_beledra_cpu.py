"""Beledra on the CPU statements of its kernels: configuration, weights, scheduling, caches and batches against the plain
oracle (the kernels themselves: tests/test_gpu_beledra.py)."""
import json
import math
import warnings

import pytest
import torch

import beledra_helpers as H
import beledra_oracle as O
from llm_systems_from_scratch_b200.models import mixers
from llm_systems_from_scratch_b200.models.beledra import BUCKETS, Beledra, BeledraConfig, RandomTensors, tensor_shapes
from llm_systems_from_scratch_b200.models.registry import build_model, load_model, model_class
from llm_systems_from_scratch_b200.ops import mixer_ops as mo
from llm_systems_from_scratch_b200.serving import Request, ServingEngine
from llm_systems_from_scratch_b200.serving.batch import StepBatch
from llm_systems_from_scratch_b200.serving.kv_cache import LayerCache, PagedSpec, SharedSpec, StateSpec
from llm_systems_from_scratch_b200.utils import safetensors as st

CPU = dict(dtype=torch.float32, device="cpu")


def model(cfg, ts):
    return Beledra(H.settings(cfg), ts, **CPU)


def engine(cfg, ts, **kw):
    args = dict(num_pages=24, page_size=4, max_batch=3, max_context=96)
    args.update(kw)
    return ServingEngine(model(cfg, ts), **args)


# --------------------------------------------------------------------------- configuration and weights
def test_configuration_is_read_and_checked():
    cfg = H.settings(H.CONFIGS["odd"])
    c = BeledraConfig.from_dict(cfg)
    assert [la.type for la in c.layers] == ["mlstm", "attention", "attention_2", "attention", "attention_2", "mlstm"]
    assert c.layers[2].mixer["kv_from"] is None and c.layers[4].mixer["kv_from"] == 2 and c.eps == 1e-4 and c.layers[3].mlp is None
    la = cfg["layers"]
    mix = lambda i, **kw: {**la[i], "mixer": {**la[i]["mixer"], **kw}}
    bad = ([{**la[0], "type": "convolution"}], [mix(0, gate_cap=1.0) | {"mlp": {"kind": "moe", "ff": 3}}], [mix(1, kv_heads=4)],
           [mix(1, mask={"size": 0})], [mix(4)], [la[0], mix(4, kv_from=0)], [*la[:4], mix(4, kv_from=4)],
           [*la[:5], mix(4, kv_from=4)], [*la[:4], mix(4, kv_heads=3)], [*la[:4], mix(4, dim=12)], [{"type": "mlstm", "mixer": {"heads": 2}}])
    for layers in bad:
        with pytest.raises(ValueError):
            BeledraConfig.from_dict({**cfg, "layers": layers})
    with warnings.catch_warnings():
        warnings.simplefilter("error")
        with pytest.raises(UserWarning):
            BeledraConfig.from_dict({**cfg, "something": 1})
    plain = mix(2, rot={"base": 100.0, "dims": 4})
    assert BeledraConfig.from_dict({**cfg, "layers": [plain]}).layers[0].mixer["rot"]["scaling"] is None
    assert model_class(cfg) is Beledra


def test_weights_are_checked_against_the_configuration():
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    shapes = tensor_shapes(BeledraConfig.from_dict(H.settings(cfg)))
    assert {k: tuple(v.shape) for k, v in ts.items() if not k.endswith(".rel")} == {k: v for k, v in shapes.items() if not k.endswith(".rel")}
    assert "l4.mix.k" not in shapes and "l3.norm2" not in shapes and shapes["l1.mix.rel"] == (BUCKETS, 6)
    for name, wrong in (("l2.mix.k", ts["l2.mix.k"][:-1]), ("l1.mix.rel", ts["l1.mix.rel"][:, :-1]), ("l0.mix.i.b", ts["l0.mix.i.b"][:-1]),
                        ("l2.mix.lq1", ts["l2.mix.lq1"][:-1]), ("l0.norm1", ts["l0.norm1"][:-1]), ("l1.mlp.down", ts["l1.mlp.down"].t())):
        with pytest.raises(ValueError):
            model(cfg, {**ts, name: wrong})
    rnd = RandomTensors(H.settings(cfg), 5)
    assert all(tuple(rnd[n].shape) == shapes[n] for n in rnd.keys())
    assert torch.equal(rnd["head"], RandomTensors(H.settings(cfg), 5)["head"])
    eng = ServingEngine(build_model(H.settings(cfg), 1, **CPU), num_pages=4, page_size=4, max_batch=1, max_context=16)
    assert len(eng.generate([[1, 2, 3]], 4)[0]) == 4


def test_folder_loads_through_the_registry(tmp_path):
    cfg, ts = H.CONFIGS["difference only"], H.tensors(H.CONFIGS["difference only"])
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(H.settings(cfg)))
    seq = H.prompts(cfg, [9])[0]
    eng = ServingEngine(load_model(str(tmp_path), **CPU), num_pages=8, page_size=4, max_batch=1, max_context=32)
    assert H.error(H.feed(eng, [seq], [[(0, 9)]])[0], H.expected(cfg, ts, [seq])[0]) < 1e-4


def test_a_shared_layer_has_no_pool_of_its_own():
    specs = [PagedSpec(8), StateSpec((2, 3)), SharedSpec(0)]
    cache = LayerCache(specs, 3, 4, 2, "cpu", torch.float32)
    assert cache.entries[2] is cache.entries[0] and LayerCache.bytes_per_page(specs, 4, 2) == 64
    m = model(H.CONFIGS["odd"], H.tensors(H.CONFIGS["odd"]))
    assert [type(layer.mixer.cache_spec()).__name__ for layer in m.runs] == [
        "StateSpec", "PagedSpec", "PagedSpec", "PagedSpec", "SharedSpec", "StateSpec"]


# ----------------------------------------------------------------------------------------- mechanisms
def test_distance_buckets():
    for rows, far in ((32, 300), (6, 14), (8, 100), (5, 33), (16, 128)):
        got = [mixers.distance_bucket(n, rows, far) for n in range(3 * far)]
        assert got == [O.distance_bucket(n, rows, far) for n in range(3 * far)]
        assert got[:rows // 2] == list(range(rows // 2)) and got == sorted(got) and got[far] == got[-1] == rows - 1
    # the second half grows by equal factors: 8 rows up to 64 tokens double the distance with every row
    assert [mixers.distance_bucket(n, 8, 64) for n in (3, 4, 7, 8, 15, 16, 31, 32, 63, 64, 1000)] == [3, 4, 4, 5, 5, 6, 6, 7, 7, 7, 7]
    rel = torch.randn(6, 3)
    for window in (1, 4, 9, 100):
        t = mixers.distance_table(rel, 14, window)
        assert t.shape[1] <= window
        for d in range(window):
            assert torch.equal(t[:, min(d, t.shape[1] - 1)], rel[O.distance_bucket(d, 6, 14)])


@pytest.mark.parametrize("dims,base,scaling", [(20, 20000.0, H.yarn(5.0, 1000, 20.0, 1.5)), (6, 500.0, H.yarn()), (16, 100.0, None),
                                               (8, 10.0, H.yarn(2.0, 4, 1.0, 0.5)), (64, 1e6, H.yarn(16.0, 8192, 64.0, 2.0))])
def test_rotation_tables(dims, base, scaling):
    table = mixers.RotaryTable(base, dims, "cpu", scaling)
    table.resize(3000)
    freq, gain = O.yarn({"dims": dims, "base": base, "scaling": scaling})
    for i, f in enumerate(freq):
        for p in (0, 1, 777, 2999):
            assert abs(float(table.table[0, p, i]) - gain * math.cos(p * f)) < 1e-6
            assert abs(float(table.table[1, p, i]) - gain * math.sin(p * f)) < 1e-6
    if dims == 20:               # fast pairs keep their frequency, slow ones are divided by the factor
        assert freq[0] == 1.0 and abs(freq[-1] * 5.0 - base ** (-18 / 20)) < 1e-12 and abs(gain - (1 + 0.1 * math.log(5))) < 1e-12


def test_matrix_memory_statement_against_its_definition():
    """Without the running maximum, in double precision: S_t = sum of decayed outer products."""
    g = torch.Generator().manual_seed(0)
    T, Hh, D, E = 40, 2, 6, 5
    q, k, v = (torch.randn(T, Hh, n, generator=g, dtype=torch.float64) for n in (D, D, E))
    i = 2 * torch.randn(T, Hh, generator=g, dtype=torch.float64)
    f = torch.nn.functional.logsigmoid(1 + 2 * torch.randn(T, Hh, generator=g, dtype=torch.float64))
    got = O.mlstm_scan(q, k, v, i, f)
    F = f.cumsum(0)
    for t in range(T):
        w = torch.exp(F[t] - F[:t + 1] + i[:t + 1]) * (k[:t + 1] * q[t]).sum(-1)           # (t + 1, heads)
        m = torch.maximum(F[t], (F[t] - F[:t + 1] + i[:t + 1]).max(0).values)              # the maximum starts at zero
        low = torch.maximum((w.sum(0) * torch.exp(-m)).abs(), torch.exp(-m)) + 1e-6
        assert torch.allclose(got[t], torch.einsum("sh,she->he", w * torch.exp(-m), v[:t + 1]) / low[:, None], atol=1e-10)


def test_residual_and_feed_forward_statements():
    g = torch.Generator().manual_seed(0)
    emb, w, y = torch.randn(11, 7, generator=g), torch.randn(7, generator=g), torch.randn(4, 7, generator=g)
    x = torch.empty(4, 7)
    h = mo.add_normed(x, tokens=torch.tensor([3, 3, 10, 0]), embed=emb)
    assert torch.equal(x, emb[[3, 3, 10, 0]]) and torch.equal(h, x)
    want = x + O.rms_norm(y, w, 1e-3)
    assert torch.allclose(mo.add_normed(x, y, w, 1e-3), want) and torch.allclose(x, want)
    gate, up = torch.randn(5, 7, generator=g), torch.randn(5, 7, generator=g)
    got = mo.glu(x, mo.padded_weight(torch.cat((gate, up)), torch.float32, "cpu"), 5, "relu")
    assert torch.allclose(got @ torch.eye(5), O.relu_glu(x, gate, up, torch.eye(5)), atol=1e-5)


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
    (tmp_path / "config.json").write_text(json.dumps(H.settings(cfg)))
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
    (tmp_path / "config.json").write_text(json.dumps(H.settings(cfg)))
    prompt = H.prompts(cfg, [6])[0]
    generate.main(["--model", str(tmp_path), "--dtype", "float32", "--device", "cpu", "--temperature", "0", "--max-tokens", "5",
                   "--prompt-ids", ",".join(map(str, prompt))])
    assert capsys.readouterr().out.strip() == ",".join(map(str, _greedy(cfg, ts, prompt, 5)))
    if torch.cuda.is_available():
        return
    (tmp_path / "s.yaml").write_text(json.dumps({"model": H.settings(cfg), "serving": {
        "max_batch": 3, "max_context": 48, "num_requests": 5, "prompt_len": [2, 20], "output_len": [2, 6], "page_size": 4}}))
    serve.main(["--config", str(tmp_path / "s.yaml"), "--offline"])
    rec = json.loads(capsys.readouterr().out.strip().splitlines()[-1])
    assert rec["requests"] == 5 and rec["model"] == "Beledra" and rec["output_tokens"] > 0


def test_serving_configuration_and_kernel_sources():
    import os
    from llm_systems_from_scratch_b200 import build_ext
    from llm_systems_from_scratch_b200.models.registry import MODELS
    from llm_systems_from_scratch_b200.utils.config import load_config, validate
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cfg = validate(load_config(os.path.join(root, "configures", "serve_beledra.yaml")), require_dataset=False)
    layers = BeledraConfig.from_dict(cfg["model"]).layers
    assert len(layers) == 24 and all(la.mixer.get("kv_from") in (None, i - 2) for i, la in enumerate(layers))
    names = {s.name for s in build_ext.sources()}
    assert build_ext.MIXERS <= names
    assert all(set(getattr(m, "KERNELS", None) or ()) <= build_ext.MIXERS for m in MODELS.values())
