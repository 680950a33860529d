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


# ------------------------------------------------------------------------------------ latent attention
def paged(latents, page, extra=5, seed=0):
    """Put every sequence's latents (T, width) on shuffled pages; unused cache rows are NaN.  -> (cache, tables)"""
    width, pages = latents[0].shape[1], [-(-len(x) // page) for x in latents]
    order = torch.randperm(sum(pages) + extra, generator=torch.Generator().manual_seed(seed)).tolist()
    cache = torch.full((sum(pages) + extra, page, width), float("nan"), dtype=latents[0].dtype, device="cuda")
    tables = torch.full((len(latents), max(pages) + 1), 10 ** 6, dtype=torch.int32)
    for i, x in enumerate(latents):
        mine = [order.pop() for _ in range(pages[i])]
        tables[i, :len(mine)] = torch.tensor(mine)
        for t in range(len(x)):
            cache[mine[t // page], t % page] = x[t]
    return cache, tables.cuda()


def stand_out(latents, q, pos, window, heads, width):
    """Make the token just inside the window agree with the query, and the one just outside it far more so."""
    c = latents[pos].new_zeros(0)
    for back, gain in ((window - 1, 3.0), (window, 9.0)):
        if 0 <= pos - back < len(latents):
            latents[pos - back] = gain * q.view(heads, width)[0] / q.view(heads, width)[0].norm() * width ** 0.5
    return c


@pytest.mark.parametrize("width,heads,window,page", [(24, 3, 7, 4), (128, 16, 44, 16), (72, 6, 33, 16), (136, 20, 64, 16),
                                                     (256, 8, 1, 16), (512, 17, 300, 16), (512, 16, 0, 64), (8, 40, 65, 5),
                                                     (384, 33, 130, 8), (512, 5, 129, 32), (256, 64, 128, 128)])
@pytest.mark.parametrize("splits", [0, 1, 3])
def test_latent_decode_at_every_edge(width, heads, window, page, splits):
    mo = mops()
    lens = [1, 2, 15, 16, 17, 32, 33, 63, 64, 65, 97, 331]
    scale = 2.0 * width ** -0.5
    q = randn(len(lens), heads * width, seed=1, dtype=BF, scale=0.5)
    lat = [randn(n, width, seed=10 + n, dtype=BF) for n in lens]
    for i, n in enumerate(lens):
        if window:
            stand_out(lat[i], q[i], n - 1, window, heads, width)
    cache, tables = paged(lat, page)
    pos = torch.tensor([n - 1 for n in lens], dtype=torch.int32, device="cuda")
    slots = torch.zeros(len(lens), dtype=torch.int64, device="cuda")
    slots[4] = -1
    got = [mo.latent_decode(q, cache, pos, slots, tables, heads, window, scale, splits, k)
           for k in ("mma", *(("tcgen05",) if width % 128 == 0 else ()))]
    rows = mo.latent_attention_rows(q, cache, None, pos, slots, tables, heads, window, scale)
    for i, n in enumerate(lens):
        if i == 4:
            assert all(float(g[i].abs().sum()) == 0.0 for g in (*got, rows))
            continue
        c = lat[i].double().cpu()[:, None, :].expand(n, heads, width)
        qs = torch.zeros(n, heads, width, dtype=torch.float64)
        qs[-1] = q[i].double().cpu().view(heads, width)
        want = O.window_attention(qs, c, c, scale, window or 10 ** 6)[-1].reshape(-1)
        for g in got:
            close(g[i], want, 1.5e-2)
        close(rows[i], want, 1e-2)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_rows_of_portions(dtype):
    """The general kernel: rows of several sequences, each with its own position and line of the tables."""
    mo = mops()
    width, heads, window, lens = 24, 5, 6, [9, 30]
    lat = [randn(n, width, seed=n, dtype=dtype) for n in lens]
    cache, tables = paged(lat, 4)
    q = randn(sum(lens), heads * width, seed=3, dtype=dtype)
    seq = torch.tensor([0] * 9 + [1] * 30, dtype=torch.int32, device="cuda")
    pos = torch.cat([torch.arange(n) for n in lens]).int().cuda()
    got = mo.latent_attention_rows(q, cache, seq, pos, torch.zeros(39, dtype=torch.int64, device="cuda"), tables, heads, window, 0.3)
    at = 0
    for i, n in enumerate(lens):
        c = lat[i].double().cpu()[:, None, :].expand(n, heads, width)
        want = O.window_attention(q[at:at + n].double().cpu().view(n, heads, width), c, c, 0.3, window)
        close(got[at:at + n], want.reshape(n, -1), 1e-2 if dtype == BF else 1e-5)
        at += n


@pytest.mark.parametrize("dh,vdim,heads", [(64, 64, 2), (64, 20, 3), (128, 128, 2), (128, 72, 1)])
@pytest.mark.parametrize("window", [0, 1, 45, 127, 128, 129, 300])
def test_window_attention_of_portions(dh, vdim, heads, window):
    """Portions of unequal length, some with earlier tokens in front; one key just inside and one just outside the last
    query's window stand out."""
    mo = mops()
    spans = [(0, 1), (0, 130), (37, 2), (500, 300), (200, 257), (1, 128)]        # (start, tokens)
    scale, qs, ks, vs, cu_q, cu_k, want = 1.3 * dh ** -0.5, [], [], [], [0], [0], []
    for i, (start, n) in enumerate(spans):
        first = max(0, start - window + 1) if window else 0
        total = start + n
        q, k, v = (randn(total, heads, d, seed=20 * i + j, dtype=BF) for j, d in enumerate((dh, dh, vdim)))
        if window:
            for back, gain in ((window - 1, 2.0), (window, 4.0)):
                if total - 1 - back >= 0:
                    k[total - 1 - back] = gain * q[-1] / q[-1].float().norm(dim=-1, keepdim=True).to(BF) * dh ** 0.5
        want.append(O.window_attention(q.double().cpu(), k.double().cpu(), v.double().cpu(), scale, window or 10 ** 6)[start:].reshape(n, -1))
        qs.append(q[start:].reshape(n, -1))
        ks.append(k[first:].reshape(total - first, -1))
        pad = torch.zeros(total - first, heads, dh, dtype=BF, device="cuda")
        pad[..., :vdim] = v[first:]
        vs.append(pad.view(total - first, -1))
        cu_q.append(cu_q[-1] + n)
        cu_k.append(cu_k[-1] + total - first)
    q, kv = torch.cat(qs), torch.cat([torch.cat(ks), torch.cat(vs)], 1)
    dev = lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")
    wide = randn(q.shape[0], heads * vdim + 3, seed=7, dtype=BF)
    for gate in (None, wide[:, 3:]):
        out = mo.rows_buffer(q.shape[0], heads * vdim, BF, "cuda")
        mo.window_attention(q, kv, dev(cu_q), dev(cu_k), 300, heads, dh, vdim, window, scale, out, gate)
        ref = torch.cat(want) * (1.0 if gate is None else torch.sigmoid(gate.double().cpu()))
        close(out, ref, 2e-2)


# --------------------------------------------------------------------------------------------- retention
def rope_table(n, base, dims):
    f = base ** (-2.0 * torch.arange(dims // 2, dtype=torch.float64) / dims)
    a = torch.outer(torch.arange(n, dtype=torch.float64), f)
    return torch.stack((a.cos(), a.sin())).float().contiguous().cuda() if dims else None


def retention_case(lens, heads, dim, vdim, dims, decay, dtype, start_states=None, seed=0):
    """Whole sequences of (start + n) tokens by the oracle -> rows of the last n tokens and the final states."""
    width = 2 * heads * (dim + vdim)
    proj = [randn(n, width, seed=seed + i, dtype=dtype) for i, n in enumerate(lens)]
    outs, states = [], []
    for p in proj:
        n, hd, he = len(p), heads * dim, heads * vdim
        x, pos = p.double().cpu(), torch.arange(len(p))
        q = O.rotate_half(x[:, :hd].reshape(n, heads, dim), pos, 1000.0, dims)
        k = O.rotate_half(x[:, hd:2 * hd].reshape(n, heads, dim), pos, 1000.0, dims) * dim ** -0.5
        v, g = x[:, 2 * hd:2 * hd + he].reshape(n, heads, vdim), x[:, 2 * hd + he:]
        o = O.rms(O.retention_scan(q, k, v, decay), 1e-4).reshape(n, he)
        outs.append(o * g * torch.sigmoid(g))
        d = torch.tensor(decay, dtype=torch.float64)
        w = d[None, :] ** (n - 1 - pos[:, None]).double()
        states.append(torch.einsum("th,thd,the->hde", w, k, v))
    return proj, outs, states


CASES = [(3, 10, 7, 6, [0.9, 0.5, 0.99]), (3, 64, 64, 48, [0.99, 0.96875, 0.95]), (3, 48, 24, 16, [0.9, 0.97, 0.995]),
         (1, 128, 128, 128, [0.9985]), (2, 128, 72, 0, [0.85, 1.0]), (1, 16, 136, 16, [0.75]),
         (1, 40, 96, 32, [0.97]), (14, 128, 128, 96, [0.9 + 0.007 * i for i in range(14)])]


@pytest.mark.parametrize("heads,dim,vdim,dims,decay", CASES)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_retention_token_by_token_and_in_portions(heads, dim, vdim, dims, decay, dtype):
    """Cut at every kind of place: the recurrent kernel, the decode kernel and - where the sizes allow it - the chunked kernel,
    one after the other on the same states."""
    mo = mops()
    lens = [1, 2, 127, 128, 129, 300]
    proj, outs, states = retention_case(lens, heads, dim, vdim, dims, decay, dtype)
    table, dev = rope_table(320, 1000.0, dims), lambda a: torch.tensor(a, dtype=torch.int32, device="cuda")
    dec = torch.tensor(decay, device="cuda")
    powers = mo.retention_powers(decay, "cuda") if mo.chunkable(dtype, dim, vdim, dims) else None
    assert (powers is None) == (dtype == F32 or dim % 8 != 0 or vdim % 8 != 0 or vdim > 128 or min(decay) < 0.8)
    tol = 1.5e-2 if dtype == BF else 5e-5

    def run(kind, state, parts):
        """parts: (sequence, start, tokens), all of one step"""
        rows = torch.cat([proj[i][a:a + n] for i, a, n in parts])
        src = mo.rows_buffer(rows.shape[0], rows.shape[1], dtype, "cuda")
        src.copy_(rows)
        pos = torch.cat([torch.arange(a, a + n) for _, a, n in parts]).int().cuda()
        slots = dev([len(lens) - i for i, _, _ in parts])
        cu = dev([0] + list(torch.tensor([n for _, _, n in parts]).cumsum(0)))
        y = mo.rows_buffer(rows.shape[0], heads * vdim, dtype, "cuda")
        if kind == "chunked":
            mo.retention_chunked(src, state, slots, cu, pos, table, powers, heads, dim, vdim, dims, 1e-4, y)
        else:
            mo.retention(src, state, slots, cu if kind == "recurrent" else None, None, pos, table, dec, heads, dim, vdim, dims, 1e-4, y)
        at = 0
        for i, a, n in parts:
            close(y[at:at + n], outs[i][a:a + n], tol)
            at += n

    everything = [(i, 0, n) for i, n in enumerate(lens)]
    for kind in ("recurrent", "chunked") if powers is not None else ("recurrent",):
        state = torch.full((len(lens) + 2, heads, dim, vdim), float("nan"), device="cuda")
        run(kind, state, everything)
        for i, s in enumerate(states):
            close(state[len(lens) - i], s, 1e-4)
        assert torch.isnan(state[0]).all() and torch.isnan(state[len(lens) + 1]).all()      # nobody's slots
        state.fill_(float("nan"))
        run("recurrent", state, [(2, 0, 3), (5, 0, 2)])
        run(kind, state, [(5, 2, 131), (2, 3, 5)])
        run("step", state, [(2, 8, 1), (5, 133, 1)])
        run(kind, state, [(2, 9, 118), (5, 134, 40)])
        run("step", state, [(5, 174, 1)])
        run(kind, state, [(5, 175, 125)])
        close(state[len(lens) - 5], states[5], 1e-4)
        close(state[len(lens) - 2], states[2], 1e-4)


def test_retention_remembers_a_far_token():
    """One token 250 positions back carries nearly all of the state; a lost or wrongly decayed state shows at once."""
    mo = mops()
    decay, n = [0.9985], 260
    proj = randn(n, 4 * 64, seed=1, dtype=BF, scale=0.05)
    proj[3, 64:128], proj[3, 128:192] = 8.0, 5.0
    proj[:, 192:] *= 30.0
    x = proj.double().cpu()
    q, k, v, g = (x[:, 64 * i:64 * i + 64].reshape(n, 1, 64) for i in range(4))
    o = O.rms(O.retention_scan(q, k * 64 ** -0.5, v, decay), 1e-6)
    want = (o * g * torch.sigmoid(g)).reshape(n, 64)
    for kind in ("chunked", "recurrent"):
        state, y = torch.zeros(1, 1, 64, 64, device="cuda"), torch.empty(n, 64, device="cuda", dtype=BF)
        pos, zero = torch.arange(n, dtype=torch.int32, device="cuda"), torch.zeros(1, dtype=torch.int32, device="cuda")
        cu = torch.tensor([0, n], dtype=torch.int32, device="cuda")
        if kind == "chunked":
            mo.retention_chunked(proj, state, zero, cu, pos, None, mo.retention_powers(decay, "cuda"), 1, 64, 64, 0, 1e-6, y)
        else:
            mo.retention(proj, state, zero, cu, None, pos, None, torch.tensor(decay, device="cuda"), 1, 64, 64, 0, 1e-6, y)
        close(y, want, 1e-2)
        assert float(state.abs().max()) > 3


# -------------------------------------------------------------------------------- sampling from fp32 logits
def test_fp32_logits_argmax_and_top_k():
    from llm_systems_from_scratch_b200.ops import native
    x = randn(40, 1003, seed=1)
    x[3, 700] = x[3, 20] = 9.0
    assert torch.equal(native.argmax_rows(x), x.argmax(-1)) and int(native.argmax_rows(x)[3]) == 20
    assert torch.equal(native.argmax_rows(x, 500), x[:, :500].argmax(-1))
    u = torch.rand(40, generator=torch.Generator().manual_seed(0)).cuda()
    for top_k in (None, 1, 5, 400):
        got = native.sample_topk(x, u, 0.7, top_k)
        ref = x.double()
        if top_k:
            ref = ref.masked_fill(ref < ref.topk(top_k, -1).values[:, -1:], float("-inf"))
        p = torch.softmax(ref / 0.7, -1)
        cdf = p.cumsum(-1)
        lo = cdf.gather(1, got[:, None]).squeeze(1) - p.gather(1, got[:, None]).squeeze(1)
        assert (p.gather(1, got[:, None]) > 0).all()
        assert ((lo - 1e-4 <= u) & (u <= lo + p.gather(1, got[:, None]).squeeze(1) + 1e-4)).all()


# ------------------------------------------------------------------------------------------- whole models
TOL = {F32: 3e-5, BF: 0.06}


def engine(cfg, ts, dtype, **kw):
    from llm_systems_from_scratch_b200.models.tedirax import Tedirax
    from llm_systems_from_scratch_b200.serving import ServingEngine
    args = dict(num_pages=64, page_size=16, max_batch=4, max_context=512, use_cuda_graphs=False)
    args.update(kw)
    return ServingEngine(Tedirax(cfg, ts, dtype, "cuda"), **args)


@pytest.mark.parametrize("dtype", [F32, BF])
@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_models_in_every_cut_and_company(name, dtype):
    """Whole prompts, token by token, portions down to two tokens, and mixed batches that leave and return, on pages and slots
    that are used again (and poisoned in between), all against the oracle on the whole sequence."""
    cfg = H.CONFIGS[name]
    ts = H.tensors(cfg)
    seqs = H.prompts(cfg, [170, 33, 1, 64, 90, 130])
    n = [len(s) for s in seqs]
    want = H.expected(cfg, ts, seqs)
    eng = engine(cfg, ts, dtype)
    whole = [[(i, k)] for i, k in enumerate(n)]
    for schedule in (whole, sum([H.alone(i, n[i], [n[i] - 40, *[1] * 40] if n[i] > 60 else [1]) for i in range(6)], []),
                     sum([H.alone(i, n[i], [2, 3, 16, 31]) for i in range(6)], []),
                     H.mixed(n, [[50, *[1] * 12], [2], [7, 1, 1], [64, 1], [15, 17, 2, 1]], live=4),
                     [[(0, 100), (1, 33), (3, 64), (4, 90)], [(5, 130), (0, 70), (2, 1)]]):
        got = H.feed(eng, seqs, schedule, poison=True)
        for i in range(6):
            assert H.error(got[i], want[i]) < TOL[dtype], (i, schedule[:3])
        assert eng.cache.allocator.free == 64 and eng.cache.slot_allocator.free == 4


@pytest.mark.parametrize("heads", [8, 20])
def test_a_large_batch_decodes_on_the_token_tiles(heads):
    """Enough requests for the tcgen05 decode kernel, which small batches do not use; a page holds more than one window."""
    cfg = H.config(90, 48, [H.latent(heads, 24, 16, 40, 128, 30, mlp=H.moe(16, 3, 2)), H.retention(2, 16, 16, [0.98, 0.9])])
    ts = H.tensors(cfg)
    lens = [5 + (7 * i) % 90 for i in range(70)]
    seqs = H.prompts(cfg, lens)
    want = H.expected(cfg, ts, seqs)
    eng = engine(cfg, ts, BF, num_pages=160, page_size=64, max_batch=70)
    steps = [[(i, n - 4) for i, n in enumerate(lens)]] + [[(i, 1) for i in range(70)]] * 4
    for g, w in zip(H.feed(eng, seqs, steps, poison=True), want):
        assert H.error(g[-4:], w[-4:]) < 0.03         # (a first token whose q.k is near zero is noise in bf16)


def test_long_decoding_stays_exact():
    cfg = H.CONFIGS["tiles"]
    ts = H.tensors(cfg)
    seq = H.prompts(cfg, [420])
    want = H.expected(cfg, ts, seq)[0]
    for dtype in (F32, BF):
        got = H.feed(engine(cfg, ts, dtype), seq, H.alone(0, 420, [5, *[1] * 415]))[0]
        assert H.error(got, want) < TOL[dtype]


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_greedy_generation_through_the_engine(dtype, graphs):
    """More requests than rows, prompts in portions, captured decode steps; every token is the oracle's choice given the tokens
    before it, unless the two best logits are closer than the precision."""
    cfg = H.CONFIGS["tiles"]
    ts = H.tensors(cfg)
    ps = H.prompts(cfg, [3, 150, 1, 40, 64, 17, 90])
    eng = engine(cfg, ts, dtype, max_batch=3, max_prefill_tokens=64, use_cuda_graphs=graphs)
    outs = eng.generate(ps, 24)
    o = O.Oracle(cfg, ts)
    sure = 0
    for p, out in zip(ps, outs):
        logits = o.logits(p + out)[len(p) - 1:-1]
        best = logits.max(-1).values
        gap = best - logits[torch.arange(len(out)), torch.tensor(out)]
        scale = (logits - logits.mean(-1, keepdim=True)).pow(2).mean(-1).sqrt()
        assert len(out) == 24 and float((gap / scale).max()) < (1e-4 if dtype == F32 else 0.15)
        sure += int((gap == 0).sum())
    assert sure > 0.9 * 24 * len(ps)
    assert eng.cache.allocator.free == eng.cache.num_pages and eng.cache.slot_allocator.free == 3
    again = eng.generate(ps[::-1], 24)[::-1]                 # other rows, pages and slots
    same = sum(a == b for x, y in zip(outs, again) for a, b in zip(x, y))
    assert same == 24 * len(ps) if dtype == F32 else same > 0.7 * 24 * len(ps)
    torch.manual_seed(0)
    drawn = eng.generate(ps[:3], 8, temperature=0.8, top_k=5)
    assert all(0 <= t < cfg["vocab"] for d in drawn for t in d)


def test_blocking_decode_step_and_graph_capture_leave_states_alone():
    """The first decode of a bucket captures its graph with a warm-up run: a recurrent state must advance once, not twice."""
    cfg = H.CONFIGS["retention only"]
    ts = H.tensors(cfg)
    p = H.prompts(cfg, [20, 9])
    want = [engine(cfg, ts, F32).generate([x], 6)[0] for x in p]
    eng = engine(cfg, ts, F32, use_cuda_graphs=True)
    from llm_systems_from_scratch_b200.serving import Request
    reqs = [Request(i, x, 6) for i, x in enumerate(p)]
    for r in reqs:
        eng.sched.add(r)
    for r in eng.sched.admit(float("inf")):
        eng.sched.start([r])
    for r, t in zip(reqs, eng.prefill(reqs).tolist()):
        r.output.append(t)
    for _ in range(5):
        for r, t in zip(reqs, eng.decode(reqs)):
            r.output.append(t)
    assert [r.output for r in reqs] == want


def test_trace_command_runs_on_the_gpu(tmp_path):
    import json
    import os
    import subprocess
    import sys
    from llm_systems_from_scratch_b200.utils import safetensors as st
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    a = H.prompts(cfg, [30])[0]
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:20], "want": [0, 19]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": a[20:], "want": [9]}], "end": ["x"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    run = subprocess.run([sys.executable, os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path), "--dtype", "float32",
                          "--out", str(tmp_path), "--max-tokens", "64"], input="\n".join(map(json.dumps, steps)) + "\n",
                         capture_output=True, text=True, timeout=300)
    assert run.returncode == 0, run.stderr[-2000:]
    assert [x for x in run.stdout.split("\n") if x.startswith("done")] == ["done 0", "done 1"]
    want = H.expected(cfg, ts, [a])[0]
    got = [torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=F32).view(-1, cfg["vocab"]) for i in (0, 1)]
    assert H.error(torch.cat(got), want[[0, 19, 29]]) < 3e-5
