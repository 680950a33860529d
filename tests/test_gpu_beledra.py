"""Beledra on the GPU: every kernel against the plain oracle, then whole models in both precisions and in every schedule."""
import pytest
import torch

import beledra_helpers as H
import beledra_oracle as O

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


def dev(a, dtype=torch.int32):
    return torch.tensor(a, dtype=dtype, device="cuda")


def padded(t):
    """The same rows with the pitch the products have."""
    out = mops().rows_buffer(t.shape[0], t.shape[1], t.dtype, "cuda")
    out.copy_(t)
    return out


# --------------------------------------------------------------------- residual stream, gated feed-forward
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("d", [5, 44, 320, 2048, 9000])
def test_add_normed(dtype, d):
    mo = mops()
    emb, w, y = randn(31, d, seed=1, dtype=dtype), randn(d, seed=2, dtype=dtype), padded(randn(9, d, seed=3, dtype=dtype))
    tok = dev([0, 30, 4, 4, 9, 1, 2, 3, 30], torch.int64)
    x = torch.full((9, d), float("nan"), device="cuda")
    h = mo.add_normed(x, tokens=tok, embed=emb)
    assert torch.equal(x, emb[tok].float()) and torch.equal(h, emb[tok])
    want = x.double() + O.rms_norm(y.double(), w.double(), 1e-3)
    h = mo.add_normed(x, y, w, 1e-3)
    close(x, want, 3e-6)
    close(h, want, 1e-2 if dtype == BF else 3e-6)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m,n,k", [(1, 7, 5), (3, 130, 33), (129, 64, 64), (200, 77, 100), (1100, 300, 72)])
@pytest.mark.parametrize("act", ["relu", "silu"])
def test_gated_product(dtype, m, n, k, act):
    mo = mops()
    a, w = padded(randn(m, k, seed=1, dtype=dtype)), mo.padded_weight(randn(2 * n, k, seed=2, dtype=dtype, scale=k ** -0.5), dtype, "cuda")
    g, u = (a.double() @ w.double().t()).split(n, 1)
    want = (torch.relu(g) if act == "relu" else g * torch.sigmoid(g)) * u
    close(mo.glu(a, w, n, act), want, 1.5e-2 if dtype == BF else 1e-5)


# --------------------------------------------------------------------------------------- grouped attention
def shape(heads, kv, maps, dim, vdim, window, rot=0, scale=None, diff=0.0, out_scale=1.0, bias=None, eps=1e-4):
    return mops().AttentionShape(heads, kv, maps, dim, vdim, rot, 1.5 * dim ** -0.5 if scale is None else scale, window, eps, diff,
                                 out_scale, bias)


def rotary(n, base, dims, scaling=None):
    from llm_systems_from_scratch_b200.models.mixers import RotaryTable
    if not dims:
        return None
    t = RotaryTable(base, dims, "cuda", scaling)
    t.resize(n)
    return t.table


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,kv,maps,dim,vdim,rot", [(4, 2, 1, 11, 9, 0), (6, 3, 2, 40, 24, 16), (2, 2, 2, 128, 72, 128), (5, 1, 1, 200, 130, 6),
                                                            (3, 3, 1, 200, 136, 112), (40, 8, 2, 24, 40, 16), (9, 3, 1, 64, 8, 0)])
def test_prepare_norms_rotates_and_appends(dtype, heads, kv, maps, dim, vdim, rot):
    """Every row at its own position; padding rows and other slots stay untouched."""
    mo = mops()
    s, scaling = shape(heads, kv, maps, dim, vdim, 8, rot), H.yarn()
    width = (heads + kv) * maps * dim + kv * vdim + 3
    proj = padded(randn(7, width, seed=1, dtype=dtype))
    wq, wk = randn(dim, seed=2, dtype=dtype), randn(dim, seed=3, dtype=dtype)
    pos, slots = dev([0, 1, 5, 90, 17, 3, 64]), dev([3, 19, -1, 0, 7, 8, 12], torch.int64)
    cache = torch.full((5, 4, s.cache_width), float("nan"), dtype=dtype, device="cuda")
    q = mo.attention_prepare(proj, s, wq, wk, rotary(100, 300.0, rot, scaling), pos, slots, cache)
    freq, gain = O.yarn({"dims": rot, "base": 300.0, "scaling": scaling}) if rot else ([], 1.0)
    x = proj.double().cpu()

    def vectors(cols, n, w):
        t = O.rms_norm(cols.reshape(7, n, dim), w.double().cpu(), s.eps)
        return O.rotate_half(t, pos.cpu(), freq, gain, rot)
    nq, nk, tol = heads * maps, kv * maps, 1e-2 if dtype == BF else 1e-5
    q = q.view(7, nq, s.q_pitch)
    close(q[..., :dim], vectors(x[:, :nq * dim], nq, wq), tol)
    assert float(q[..., dim:].abs().sum()) == 0.0
    flat, live = cache.view(20, -1), slots >= 0
    rows = flat[slots[live]]
    close(rows[:, :nk * s.k_pitch].view(6, nk, s.k_pitch)[..., :dim], vectors(x[:, nq * dim:(nq + nk) * dim], nk, wk)[live.cpu()], tol)
    v = rows[:, nk * s.k_pitch:].view(6, kv, s.v_pitch)
    assert torch.equal(v[..., :vdim].reshape(6, -1), proj[live, (nq + nk) * dim:(nq + nk) * dim + kv * vdim])
    assert int(torch.isnan(flat).any(1).sum()) == 14 and float(v[..., vdim:].abs().sum()) == 0.0
    before = cache.clone()
    again = mo.attention_prepare(proj, s, wq, None, rotary(100, 300.0, rot, scaling), pos, slots, cache)      # keys of another layer
    assert torch.equal(again.view(7, nq, -1), q) and torch.equal(cache.nan_to_num(7.0), before.nan_to_num(7.0))


def paged(rows, page, extra=5, seed=0):
    """Put every sequence's cache rows (T, width) on shuffled pages; unused cache rows are NaN.  -> (cache, tables)"""
    width, pages = rows[0].shape[1], [-(-len(x) // page) for x in rows]
    order = torch.randperm(sum(pages) + extra, generator=torch.Generator().manual_seed(seed)).tolist()
    cache = torch.full((sum(pages) + extra, page, width), float("nan"), dtype=rows[0].dtype, device="cuda")
    tables = torch.full((len(rows), max(pages) + 1), 10 ** 6, dtype=torch.int32)
    for i, x in enumerate(rows):
        mine = [order.pop() for _ in range(pages[i])]
        tables[i, :len(mine)] = torch.tensor(mine)
        for t in range(len(x)):
            cache[mine[t // page], t % page] = x[t]
    return cache, tables.cuda()


def case(s, lens, seed=0, dtype=BF, queries=1):
    """Random keys and values of some sequences and the queries of their last ``queries[i]`` positions.  In every sequence the key
    just inside the last query's window agrees with it, and the one just outside far more so.  -> q, cache rows, expected"""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *sh: torch.randn(*sh, generator=g).to(dtype)
    qs, rows, want = [], [], []
    for n, nq in zip(lens, queries if isinstance(queries, list) else [queries] * len(lens)):
        q, k, v = rnd(n, s.heads * s.maps, s.dim), rnd(n, s.kv_heads * s.maps, s.dim), rnd(n, s.kv_heads, s.vdim)
        for back, gain in ((s.window - 1, 2.0), (s.window, 5.0)):
            if n - 1 - back >= 0:
                for m in range(s.maps):
                    a = q[-1, m::s.maps][::s.heads // s.kv_heads].float()
                    k[n - 1 - back, m::s.maps] = (gain * a / a.norm(dim=-1, keepdim=True) * s.dim ** 0.5).to(dtype)
        bias = None
        if s.bias is not None:
            idx = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).clamp(0, s.bias.shape[1] - 1)
            bias = s.bias.double().cpu()[:, idx]
        o = [O.window_attention(q[:, m::s.maps].double(), k[:, m::s.maps].double(), v.double(), s.scale, s.window, bias) for m in range(s.maps)]
        o = o[0] if s.maps == 1 else O.rms(o[0] - s.difference * o[1], s.eps) * s.out_scale
        want.append(o[n - nq:].reshape(nq, -1))
        pad = lambda t, to: torch.nn.functional.pad(t, (0, to - t.shape[-1]))
        qs.append(pad(q[n - nq:], s.q_pitch).reshape(nq, -1))
        rows.append(torch.cat((pad(k, s.k_pitch).reshape(n, -1), pad(v, s.v_pitch).reshape(n, -1)), 1))
    return torch.cat(qs).cuda(), rows, torch.cat(want)


def table(heads, n, seed=9):
    return randn(heads, n, seed=seed, scale=2.0)


SHAPES = [dict(heads=3, kv=3, maps=1, dim=24, vdim=40, window=7), dict(heads=6, kv=2, maps=1, dim=64, vdim=64, window=44),
          dict(heads=12, kv=3, maps=1, dim=128, vdim=128, window=130, bias=130), dict(heads=20, kv=1, maps=1, dim=40, vdim=72, window=64, bias=5),
          dict(heads=4, kv=1, maps=1, dim=16, vdim=8, window=1, bias=1), dict(heads=8, kv=4, maps=1, dim=104, vdim=128, window=1000, scale=-0.1),
          dict(heads=4, kv=2, maps=2, dim=64, vdim=128, window=33, diff=0.7, out_scale=0.4), dict(heads=3, kv=1, maps=2, dim=24, vdim=24, window=300, diff=0.2),
          dict(heads=20, kv=1, maps=2, dim=128, vdim=96, window=128, diff=0.6, out_scale=0.5),
          dict(heads=2, kv=2, maps=2, dim=40, vdim=64, window=65, diff=-0.4, bias=40)]


def made(kw):
    kw = dict(kw)
    if kw.get("bias"):
        kw["bias"] = table(kw["heads"], kw["bias"])
    return shape(**kw)


@pytest.mark.parametrize("kw", SHAPES)
@pytest.mark.parametrize("page", [4, 64])
def test_decode_at_every_edge(kw, page):
    mo, s = mops(), made(kw)
    lens = [1, 2, 15, 16, 17, 32, 33, 63, 64, 65, 97, 331]
    q, rows, want = case(s, lens)
    cache, tables = paged([r.cuda() for r in rows], page)
    pos, slots = dev([n - 1 for n in lens]), torch.zeros(len(lens), dtype=torch.int64, device="cuda")
    slots[4] = -1
    wide = randn(len(lens), s.heads * s.vdim + 3, seed=7, dtype=BF)
    for gate in (None, wide[:, 3:]):
        ref = want * (1.0 if gate is None else torch.sigmoid(gate.double().cpu()))
        ref[4] = 0.0
        for splits in (0, 1, 3):
            out = torch.empty(len(lens), s.heads * s.vdim, dtype=BF, device="cuda")
            mo.attention_decode(q, s, cache, pos, slots, tables, out, gate, splits)
            out[4] = out[4].nan_to_num(99.0) if gate is None else out[4]
            close(out[torch.arange(len(lens)) != 4], ref[torch.arange(len(lens)) != 4], 2e-2)
        mo.attention_rows(q, s, cache, None, pos, slots, tables, out, gate)
        close(out, ref, 1.5e-2)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("kw", [dict(heads=4, kv=2, maps=1, dim=11, vdim=9, window=6, bias=4), dict(heads=3, kv=1, maps=2, dim=150, vdim=140, window=5, diff=0.3)])
def test_general_rows_of_portions(kw, dtype):
    mo, s = mops(), made(kw)
    lens = [9, 30]
    q, rows, want = case(s, lens, dtype=dtype, queries=[9, 30])
    cache, tables = paged([r.cuda() for r in rows], 4)
    seq, pos = dev([0] * 9 + [1] * 30), torch.cat([torch.arange(n) for n in lens]).int().cuda()
    out = torch.empty(39, s.heads * s.vdim, dtype=dtype, device="cuda")
    mo.attention_rows(q, s, cache, seq, pos, torch.zeros(39, dtype=torch.int64, device="cuda"), tables, out)
    close(out, want, 1.5e-2 if dtype == BF else 1e-5)


@pytest.mark.parametrize("kw", [k for k in SHAPES if k.get("scale", 1) > 0])
@pytest.mark.parametrize("page", [16, 64, 128])
def test_portions_of_prompts(kw, page):
    """Portions of unequal length, some with earlier tokens in front, cut inside tiles and pages."""
    mo, s = mops(), made(kw)
    spans = [(0, 1), (0, 130), (37, 2), (300, 290), (200, 57), (1, 128), (127, 129)]        # (start, tokens)
    q, rows, want = case(s, [a + n for a, n in spans], queries=[n for _, n in spans])
    cache, tables = paged([r.cuda() for r in rows], page)
    cu = dev([0, *torch.tensor([n for _, n in spans]).cumsum(0).tolist()])
    pos = torch.cat([torch.arange(a, a + n) for a, n in spans]).int().cuda()
    wide = randn(q.shape[0], s.heads * s.vdim + 3, seed=7, dtype=BF)
    for gate in (None, wide[:, 3:]):
        out = mo.rows_buffer(q.shape[0], s.heads * s.vdim, BF, "cuda")
        mo.attention_portions(q, s, cache, pos, cu, 290, tables, out, gate)
        close(out, want * (1.0 if gate is None else torch.sigmoid(gate.double().cpu())), 2e-2)


def test_bad_indices_are_reported_not_followed():
    from llm_systems_from_scratch_b200.ops import native
    mo, s = mops(), shape(2, 1, 1, 16, 16, 50, rot=4)
    q, out = torch.ones(2, 128, device="cuda", dtype=BF), torch.empty(2, 32, device="cuda", dtype=BF)
    cache, tables, pos = torch.zeros(3, 64, 32, device="cuda", dtype=BF), dev([[0, 7], [1, 0]]), dev([70, 2])
    slots, proj, w = torch.zeros(2, dtype=torch.int64, device="cuda"), torch.ones(2, 64, device="cuda", dtype=BF), torch.ones(16, device="cuda", dtype=BF)
    state, gates = torch.zeros(2, 2, mo.mlstm_state(16, 16), device="cuda"), torch.zeros(2, 8, device="cuda")[:, :4]
    memory = lambda slot, cu: mo.mlstm(torch.ones(2, 128, device="cuda", dtype=BF), gates, torch.zeros(4, device="cuda"), torch.ones(32, device="cuda", dtype=BF),
                                       state, dev(slot), cu, None, dev([0, 1]), 2, 16, 16, 5.0, 1e-5, out, cu is not None)
    x, emb = torch.zeros(2, 16, device="cuda"), torch.ones(4, 16, device="cuda")
    for bad in (lambda: mo.attention_decode(q, s, cache, pos, slots, tables, out), lambda: mo.attention_rows(q, s, cache, None, pos, slots, tables, out),
                lambda: mo.attention_portions(q, s, cache, dev([70, 71]), dev([0, 2]), 2, tables[:1], out),
                lambda: mo.attention_prepare(proj, s, w, w, rotary(9, 10.0, 4), dev([0, 1]), dev([0, 192], torch.int64), cache),
                lambda: mo.attention_prepare(proj, s, w, None, rotary(9, 10.0, 4), dev([0, 9]), slots, cache),
                lambda: memory([0, 2], None), lambda: memory([2], dev([0, 2])),
                lambda: mo.add_normed(x, tokens=dev([1, 4], torch.int64), embed=emb)):
        bad()
        torch.cuda.synchronize()
        with pytest.raises(native.KernelError):
            native.check_status()


# ------------------------------------------------------------------------------------ matrix memory (mLSTM)
def memory_case(lens, heads, dim, vdim, cap, dtype, seed=0, gate_scale=2.0, forget=2.0):
    """Whole sequences by the oracle: rows (q | k | v | g), gates, outputs."""
    bias = torch.cat((randn(heads, seed=90), forget + randn(heads, seed=91)))
    weight = randn(heads * vdim, seed=92, dtype=dtype)
    proj = [randn(n, 2 * heads * (dim + vdim), seed=seed + i, dtype=dtype) for i, n in enumerate(lens)]
    gates = [randn(n, 2 * heads, seed=50 + seed + i, scale=gate_scale) for i, n in enumerate(lens)]
    outs = []
    for p, gt in zip(proj, gates):
        n, hd, he = len(p), heads * dim, heads * vdim
        x, z = p.double().cpu(), gt.double().cpu() + bias.double().cpu()
        q, k = x[:, :hd].reshape(n, heads, dim) * dim ** -0.5, x[:, hd:2 * hd].reshape(n, heads, dim)
        v, g = x[:, 2 * hd:2 * hd + he].reshape(n, heads, vdim), x[:, 2 * hd + he:]
        i, f = cap * torch.tanh(z[:, :heads] / cap), torch.nn.functional.logsigmoid(cap * torch.tanh(z[:, heads:] / cap))
        o = O.rms(O.mlstm_scan(q, k, v, i, f), 1e-4).reshape(n, he)
        outs.append(o * weight.double().cpu() * torch.sigmoid(g))
    return proj, gates, bias.cuda(), weight, outs


CASES = [(3, 10, 7, 4.0), (2, 64, 64, 15.0), (3, 48, 24, 8.0), (1, 128, 128, 15.0), (2, 128, 72, 20.0), (1, 16, 136, 5.0), (2, 40, 96, 15.0),
         (1, 8, 8, 10.0), (14, 128, 128, 12.0)]


@pytest.mark.parametrize("heads,dim,vdim,cap", CASES)
@pytest.mark.parametrize("dtype", [BF, F32])
def test_memory_token_by_token_and_in_portions(heads, dim, vdim, cap, dtype):
    """Cut at every kind of place: the recurrent kernel, the decode kernel and - where the sizes allow it - the chunked kernel,
    one after the other on the same states."""
    mo = mops()
    lens = [1, 2, 127, 128, 129, 300]
    proj, gates, bias, weight, outs = memory_case(lens, heads, dim, vdim, cap, dtype)
    chunked = mo.mlstm_chunkable(dtype, dim, vdim)
    assert chunked == (dtype == BF and dim % 8 == 0 and vdim % 8 == 0 and vdim <= 128)
    tol = 2e-2 if dtype == BF else 1e-4

    def run(kind, state, parts):
        """parts: (sequence, start, tokens), all of one step"""
        src, gt = padded(torch.cat([proj[i][a:a + n] for i, a, n in parts])), padded(torch.cat([gates[i][a:a + n] for i, a, n in parts]))
        pos = torch.cat([torch.arange(a, a + n) for _, a, n in parts]).int().cuda()
        slots = dev([len(lens) - i for i, _, _ in parts])
        cu = dev([0, *torch.tensor([n for _, _, n in parts]).cumsum(0).tolist()])
        y = mo.rows_buffer(src.shape[0], heads * vdim, dtype, "cuda")
        mo.mlstm(src, gt, bias, weight, state, slots, None if kind == "step" else cu, None, pos, heads, dim, vdim, cap, 1e-4, y,
                 kind == "chunked")
        at = 0
        for i, a, n in parts:
            close(y[at:at + n], outs[i][a:a + n], tol)
            at += n

    kinds = ("recurrent", "chunked") if chunked else ("recurrent",)
    finals = []
    for kind in kinds:
        state = torch.full((len(lens) + 2, heads, mo.mlstm_state(dim, vdim)), float("nan"), device="cuda")
        run(kind, state, [(i, 0, n) for i, n in enumerate(lens)])
        assert torch.isnan(state[0]).all() and torch.isnan(state[len(lens) + 1]).all()      # nobody's slots
        finals.append(state[1:len(lens) + 1, :, :dim * vdim + dim + 1].clone())
        state.fill_(float("nan"))
        run("recurrent", state, [(2, 0, 3), (5, 0, 2)])
        run(kind, state, [(5, 2, 131), (2, 3, 5)])
        run("step", state, [(2, 8, 1), (5, 133, 1)])
        run(kind, state, [(2, 9, 118), (5, 134, 40)])
        run("step", state, [(5, 174, 1)])
        run(kind, state, [(5, 175, 125)])
        for i in (2, 5):
            close(state[len(lens) - i, :, :dim * vdim + dim + 1], finals[0][len(lens) - i - 1], 2e-4)
    close(finals[-1], finals[0], 2e-4)
    if mo.mlstm_steps(dim, vdim):                        # a step that takes the gates' products itself
        w = mo.padded_weight(randn(2 * heads, 77, seed=93, dtype=dtype, scale=0.2), dtype, "cuda")
        hin, ys = padded(randn(2, 77, seed=94, dtype=dtype)), []
        for gt in ((hin, w), hin.float() @ w.float().t()):
            st = torch.zeros(2, heads, mo.mlstm_state(dim, vdim), device="cuda")
            st[..., :dim * vdim + dim + 1] = finals[0][:2]
            ys.append(mo.rows_buffer(2, heads * vdim, dtype, "cuda"))
            mo.mlstm(padded(proj[2][:2]), gt, bias, weight, st, dev([1, 0]), None, None, dev([9, 9]), heads, dim, vdim, cap, 1e-4, ys[-1])
        close(ys[0], ys[1], 1e-2 if dtype == BF else 1e-4)
    idle = torch.zeros(2, heads, mo.mlstm_state(dim, vdim), device="cuda")
    y = torch.ones(1, heads * vdim, dtype=dtype, device="cuda")
    mo.mlstm(padded(proj[0]), padded(gates[0]), bias, weight, idle, dev([-1]), None, None, dev([0]), heads, dim, vdim, cap, 1e-4, y)
    assert float(y.abs().sum()) == 0.0 and float(idle.abs().sum()) == 0.0


@pytest.mark.parametrize("forget,scale", [(9.0, 0.1), (-9.0, 4.0), (0.0, 12.0)])
def test_memory_under_extreme_gates(forget, scale):
    """Gates that keep everything, forget everything, or jump between both; the running maximum leaves zero in both directions."""
    mo = mops()
    proj, gates, bias, weight, outs = memory_case([300], 2, 64, 40, 15.0, BF, seed=3, gate_scale=scale, forget=forget)
    for kind in ("chunked", "recurrent"):
        state, y = torch.full((1, 2, mo.mlstm_state(64, 40)), float("nan"), device="cuda"), mo.rows_buffer(300, 80, BF, "cuda")
        mo.mlstm(padded(proj[0]), padded(gates[0]), bias, weight, state, dev([0]), dev([0, 300]), None,
                 torch.arange(300, dtype=torch.int32, device="cuda"), 2, 64, 40, 15.0, 1e-4, y, kind == "chunked")
        close(y, outs[0], 2e-2)


def test_memory_keeps_a_far_token():
    """One token 250 positions back enters with a wide open gate and is kept; the later ones hardly enter."""
    mo = mops()
    n = 260
    proj, gates, bias, weight, _ = memory_case([n], 1, 64, 64, 15.0, BF, forget=0.0)
    bias.zero_()
    gates[0][:, 0], gates[0][:, 1] = -6.0, 12.0
    gates[0][3, 0] = 4.0
    x = proj[0].double().cpu()
    q, k, v, g = (x[:, 64 * i:64 * i + 64].reshape(n, 1, 64) for i in range(4))
    z = 15 * torch.tanh(gates[0].double().cpu() / 15)
    o = O.rms(O.mlstm_scan(q / 8, k, v, z[:, :1], torch.nn.functional.logsigmoid(z[:, 1:])), 1e-4)
    want = (o * torch.sigmoid(g)).reshape(n, 64) * weight.double().cpu()
    away = O.rms(O.mlstm_scan(q / 8, k, v, torch.where(torch.arange(n)[:, None] == 3, -6.0, z[:, :1]), torch.nn.functional.logsigmoid(z[:, 1:])), 1e-4)
    assert float(((away - o).reshape(n, -1)[-1]).abs().max()) > 0.5              # without that token the last row is another
    for kind in ("chunked", "recurrent"):
        state, y = torch.zeros(1, 1, mo.mlstm_state(64, 64), device="cuda"), torch.empty(n, 64, device="cuda", dtype=BF)
        mo.mlstm(proj[0], gates[0], bias, weight, state, dev([0]), dev([0, n]), None, torch.arange(n, dtype=torch.int32, device="cuda"), 1, 64, 64,
                 15.0, 1e-4, y, kind == "chunked")
        close(y, want, 2e-2)


# ------------------------------------------------------------------------------------------- whole models
# Worst row of a sequence.  In bf16 a few rows are ill-conditioned (a difference of two maps, or a sublayer's output, that nearly
# cancels is scaled up by the norm behind it), so most rows have to be far better than the worst.
TOL = {F32: 5e-5, BF: 0.3}
MOST = {F32: 5e-5, BF: 0.08}


def agrees(got, want, dtype):
    rows = torch.tensor([H.error(got[i:i + 1], want[i:i + 1]) for i in range(len(want))])
    return float(rows.max()) < TOL[dtype] and (len(rows) < 20 or float(rows.quantile(0.95)) < MOST[dtype])


def engine(cfg, ts, dtype, **kw):
    from llm_systems_from_scratch_b200.models.beledra import Beledra
    from llm_systems_from_scratch_b200.serving import ServingEngine
    args = dict(num_pages=64, page_size=16, max_batch=4, max_context=512, use_cuda_graphs=False)
    args.update(kw)
    return ServingEngine(Beledra(H.settings(cfg), ts, dtype, "cuda"), **args)


@pytest.mark.parametrize("name", list(H.CONFIGS))
def test_models_in_every_cut_and_company(name):
    """Whole prompts, token by token, portions down to two tokens, and mixed batches that leave and return, on pages and slots
    that are used again (and poisoned in between), all against the oracle on the whole sequence."""
    cfg = H.CONFIGS[name]
    ts = H.tensors(cfg)
    seqs = H.prompts(cfg, [170, 33, 1, 64, 90, 130])
    n = [len(s) for s in seqs]
    want = H.expected(cfg, ts, seqs)
    whole = [[(i, k)] for i, k in enumerate(n)]
    for dtype in (F32, BF):
        eng = engine(cfg, ts, dtype)
        for schedule in (whole, sum([H.alone(i, n[i], [n[i] - 40, *[1] * 40] if n[i] > 60 else [1]) for i in range(6)], []),
                         sum([H.alone(i, n[i], [2, 3, 16, 31]) for i in range(6)], []),
                         H.mixed(n, [[50, *[1] * 12], [2], [7, 1, 1], [64, 1], [15, 17, 2, 1]], live=4),
                         [[(0, 100), (1, 33), (3, 64), (4, 90)], [(5, 130), (0, 70), (2, 1)]]):
            got = H.feed(eng, seqs, schedule, poison=True)
            for i in range(6):
                assert agrees(got[i], want[i], dtype), (i, dtype, schedule[:3], H.error(got[i], want[i]))
            assert eng.cache.allocator.free == 64 and eng.cache.slot_allocator.free == 4


def test_a_large_batch_decodes_as_each_alone():
    cfg = H.CONFIGS["wide"]
    ts = H.tensors(cfg)
    lens = [5 + (7 * i) % 90 for i in range(70)]
    seqs = H.prompts(cfg, lens)
    eng = engine(cfg, ts, BF, num_pages=160, page_size=64, max_batch=70)
    steps = [[(i, n - 4) for i, n in enumerate(lens)]] + [[(i, 1) for i in range(70)]] * 4
    got = H.feed(eng, seqs, steps, poison=True)
    for i in range(0, 70, 9):
        assert agrees(got[i], H.expected(cfg, ts, [seqs[i]])[0], BF)


def test_long_decoding_stays_exact():
    cfg = H.CONFIGS["tiles"]
    ts = H.tensors(cfg)
    seq = H.prompts(cfg, [330])
    want = H.expected(cfg, ts, seq)[0]
    for dtype in (F32, BF):
        got = H.feed(engine(cfg, ts, dtype), seq, H.alone(0, 330, [5, *[1] * 325]))[0]
        assert agrees(got, want, dtype)


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
        assert len(out) == 24 and float((gap / scale).max()) < (1e-4 if dtype == F32 else 0.2)
        sure += int((gap == 0).sum())
    assert sure > 0.85 * 24 * len(ps)
    assert eng.cache.allocator.free == eng.cache.num_pages and eng.cache.slot_allocator.free == 3
    again = eng.generate(ps[::-1], 24)[::-1]                 # other rows, pages and slots
    same = sum(a == b for x, y in zip(outs, again) for a, b in zip(x, y))
    assert same == 24 * len(ps) if dtype == F32 else same > 0.6 * 24 * len(ps)
    torch.manual_seed(0)
    drawn = eng.generate(ps[:3], 8, temperature=0.8, top_k=5)
    assert all(0 <= t < cfg["vocab"] for d in drawn for t in d)


def test_trace_command_runs_on_the_gpu(tmp_path):
    import json
    import os
    import subprocess
    import sys
    from llm_systems_from_scratch_b200.utils import safetensors as st
    cfg = H.CONFIGS["odd"]
    ts = H.tensors(cfg)
    st.save(str(tmp_path / "model.safetensors"), ts)
    (tmp_path / "config.json").write_text(json.dumps(H.settings(cfg)))
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
    assert H.error(torch.cat(got), want[[0, 19, 29]]) < 5e-5
