"""Tedirax on the GPU: every kernel against the plain oracle, then whole models in both precisions and in every schedule."""
import pytest
import torch

import tedirax_helpers as H
import tedirax_oracle as O

pytestmark = pytest.mark.gpu
BF, F32 = torch.bfloat16, torch.float32


@pytest.fixture(autouse=True)
def status_word_stays_clean():
    yield
    from llm_systems_from_scratch_b200.ops import native
    torch.cuda.synchronize()
    native.check_status()


def mops():
    from llm_systems_from_scratch_b200.ops import mixer_ops
    return mixer_ops


def randn(*shape, seed=0, dtype=F32, scale=1.0):
    return (scale * torch.randn(*shape, generator=torch.Generator().manual_seed(seed))).to(dtype).cuda()


def close(got, want, tol):
    got, want = got.double().cpu(), want.double().cpu()
    assert not torch.isnan(got).any()
    d = float((got - want).abs().max())
    assert d <= tol * max(1.0, float(want.abs().max())), d


# ------------------------------------------------------------------------------------ matrix products
@pytest.mark.parametrize("m,n,k", [(1, 7, 5), (3, 130, 33), (128, 64, 64), (200, 77, 100), (1100, 300, 72)])
@pytest.mark.parametrize("dtype", [BF, F32])
def test_linear_of_any_size_and_accumulation(m, n, k, dtype):
    mo = mops()
    w = mo.padded_weight(randn(n, k, seed=1, dtype=dtype), dtype, "cuda")
    a = mo.rows_buffer(m, k, dtype, "cuda")
    a.copy_(randn(m, k, seed=2, dtype=dtype))
    want = a.double() @ w.double().t()
    close(mo.linear(a, w), want, 1e-2 if dtype == BF else 1e-5)
    x = randn(m, n, seed=3)
    want = x.double() + want
    mo.linear(a, w, out=x, accumulate=True)
    close(x, want, 1e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows,width,ff,experts,top", [(1, 40, 24, 3, 2), (37, 44, 13, 5, 3), (300, 128, 72, 7, 1), (700, 72, 136, 4, 4)])
def test_experts_by_table(dtype, rows, width, ff, experts, top):
    """Plan, both grouped products and the sum in the residual pass, against one expert after the other; rows with a
    negative slot take no part."""
    mo = mops()
    g = torch.Generator().manual_seed(rows)
    table = torch.stack([torch.randperm(experts, generator=g)[:top] for _ in range(50)]).int().cuda()
    tokens = torch.randint(0, 50, (rows,), generator=g).cuda()
    slots = torch.zeros(rows, dtype=torch.int64, device="cuda")
    slots[3::5] = -1
    ws = [tuple(randn(*s, seed=10 * e + i, dtype=dtype, scale=s[1] ** -0.5) for i, s in enumerate(((ff, width), (ff, width), (width, ff))))
          for e in range(experts)]
    w_gu = mo.padded_weight(torch.cat([t for e in ws for t in e[:2]]), dtype, "cuda")
    w_dn = mo.padded_weight(torch.cat([e[2] for e in ws]), dtype, "cuda")
    nw = torch.ones(width, device="cuda", dtype=dtype)
    x = randn(rows, width, seed=5)
    (pos,), (group,) = mo.moe_plan(tokens, slots, [table], [experts])
    cpu_pos, cpu_group = mo.moe_plan(tokens.cpu(), slots.cpu(), [table.cpu()], [experts])
    assert sorted(pos.flatten().tolist()) == sorted(cpu_pos[0].flatten().tolist()) and torch.equal(group.cpu(), cpu_group[0])
    before = x.clone()
    h, xg = mo.residual_norm(x, nw, 1e-6, scatter=(pos, mo.plan_tiles(rows, experts, top) * mo.TILE))
    assert torch.equal(x, before)
    hid = mo.gemm_rows(xg, w_gu, group, ff, True)
    y = mo.gemm_rows(hid, w_dn, group, width, False)
    mo.residual_norm(x, pending=(y, pos, 1.0 / top))
    live = (slots >= 0).cpu()
    want = before.double().cpu()
    add = O.table_moe(h.double().cpu(), tokens.cpu(), table.cpu(), [tuple(t.double().cpu() for t in e) for e in ws], top)
    want[live] += add[live]
    close(x, want, 2e-2 if dtype == BF else 2e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,k,n,m", [(3, 16, 24, 5), (20, 128, 136, 130), (5, 72, 9, 33)])
def test_products_per_head_and_gate(dtype, heads, k, n, m):
    mo = mops()
    a = mo.rows_buffer(m, heads * k, dtype, "cuda")
    a.copy_(randn(m, heads * k, seed=1, dtype=dtype))
    w = mo.padded_weight(randn(heads * n, k, seed=2, dtype=dtype, scale=k ** -0.5), dtype, "cuda")
    wide = randn(m, heads * n + 13, seed=3, dtype=dtype)
    gate = wide[:, 13:] if n % 8 else wide[:, 8:8 + heads * n]
    want = torch.cat([a[:, h * k:(h + 1) * k].double() @ w[h * n:(h + 1) * n].double().t() for h in range(heads)], 1)
    close(mo.gemm_heads(a, w, heads, k, n), want, 1e-2 if dtype == BF else 1e-5)
    close(mo.gemm_heads(a, w, heads, k, n, gate=gate), want * torch.sigmoid(gate.double()), 1e-2 if dtype == BF else 1e-5)


# ------------------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("d", [5, 44, 192, 1024, 4100])
def test_residual_norm(dtype, d):
    mo = mops()
    r, v, top = 9, 31, 3
    emb, w = randn(v, d, seed=1, dtype=dtype), randn(d, seed=2, dtype=dtype)
    tok = torch.tensor([0, 30, 4, 4, 9, 1, 2, 3, 30], device="cuda")
    pos = torch.randperm(128)[:r * top].view(r, top).int().cuda()
    pos[2, 1] = -1
    y = mo.rows_buffer(128, d, dtype, "cuda")
    y.copy_(randn(128, d, seed=4, dtype=dtype))
    tol = 1e-2 if dtype == BF else 1e-5
    x = torch.full((r, d), float("nan"), device="cuda")
    h, xg = mo.residual_norm(x, w, 1e-3, tokens=tok, embed=emb, scatter=(pos, 128))
    assert torch.equal(x, emb[tok].float())
    close(h, O.rms_norm(x.double(), w.double(), 1e-3), tol)
    for i in range(r):
        for k in range(top):
            if pos[i, k] >= 0:
                assert torch.equal(xg[pos[i, k]], h[i])
    add = torch.stack([sum(y[p].double() for p in row.tolist() if p >= 0) for row in pos])
    want = x.double() + 0.25 * add
    rows = torch.tensor([8, 2, 2], device="cuda")
    keep = x.clone()
    hr, _ = mo.residual_norm(x, w, 1e-3, row_index=rows, pending=(y, pos, 0.25))
    assert torch.equal(x, keep)
    close(hr, O.rms_norm(want[rows], w.double(), 1e-3), tol)
    h, _ = mo.residual_norm(x, w, 1e-3, pending=(y, pos, 0.25))
    close(x, want, 1e-6 if dtype == F32 else 1e-5)
    close(h, O.rms_norm(want, w.double(), 1e-3), tol)


def test_bad_indices_are_reported_not_followed():
    from llm_systems_from_scratch_b200.ops import native
    mo = mops()
    x, w, emb = torch.zeros(2, 16, device="cuda"), torch.ones(16, device="cuda"), torch.ones(4, 16, device="cuda")
    cache, q = torch.zeros(3, 4, 16, device="cuda", dtype=BF), torch.ones(2, 32, device="cuda", dtype=BF)
    pos, tables = torch.tensor([5, 2], dtype=torch.int32, device="cuda"), torch.tensor([[0, 7], [1, 0]], dtype=torch.int32, device="cuda")
    slots = torch.zeros(2, dtype=torch.int64, device="cuda")
    for bad in (lambda: mo.residual_norm(x, w, 1e-5, tokens=torch.tensor([1, 9], device="cuda"), embed=emb),
                lambda: mo.residual_norm(x, w, 1e-5, row_index=torch.tensor([5], device="cuda")),
                lambda: mo.latent_decode(q, cache, pos, slots, tables, 2, 0, 1.0),
                lambda: mo.latent_attention_rows(q, cache, None, pos, slots, tables, 2, 0, 1.0),
                lambda: mo.latent_norm_append(torch.ones(1, 24, device="cuda", dtype=BF), torch.ones(8, device="cuda", dtype=BF),
                                              torch.ones(16, device="cuda", dtype=BF), 1e-5, cache, torch.tensor([12], device="cuda"))):
        bad()
        torch.cuda.synchronize()
        with pytest.raises(native.KernelError):
            native.check_status()
    assert float(cache.abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("qr,kvr", [(19, 21), (64, 24), (512, 128)])
def test_latent_norm_append(dtype, qr, kvr):
    mo = mops()
    proj = mo.rows_buffer(7, qr + kvr + 10, dtype, "cuda")
    proj.copy_(randn(7, qr + kvr + 10, seed=1, dtype=dtype))
    wq, wk = randn(qr, seed=2, dtype=dtype), randn(kvr, seed=3, dtype=dtype)
    cache = torch.zeros(5, 4, mo.pitch(kvr), dtype=dtype, device="cuda")
    slots = torch.tensor([3, 19, -1, 0, 7, 8, 12], device="cuda")
    cq = mo.latent_norm_append(proj, wq, wk, 1e-3, cache, slots)
    tol = 1e-2 if dtype == BF else 1e-5
    close(cq, O.rms_norm(proj[:, :qr].double(), wq.double(), 1e-3), tol)
    want = O.rms_norm(proj[:, qr:qr + kvr].double(), wk.double(), 1e-3)
    flat = cache.view(20, -1)
    live = slots >= 0
    close(flat[slots[live], :kvr], want[live], tol)
    assert int((flat.abs().sum(1) > 0).sum()) == 6 and float(flat[:, kvr:].abs().sum()) == 0.0
