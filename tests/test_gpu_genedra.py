"""Genedra on the GPU: every kernel against the plain oracle, then whole models in both precisions and in every schedule."""
import math

import pytest
import torch

import genedra_helpers as H
import genedra_oracle as O

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


def rotary(n, base, dims, scaling=None):
    from llm_systems_from_scratch_b200.models.mixers import RotaryTable
    if not dims:
        return None
    t = RotaryTable(base, dims, "cuda", scaling)
    t.resize(n)
    return t.table


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


# ------------------------------------------------------------------------------------------ products and their ends
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m,n,k", [(1, 7, 40), (3, 130, 33), (129, 64, 64), (5, 72, 4096), (200, 77, 4168), (1100, 300, 72), (2100, 1032, 136)])
def test_products_finish_with_bias_gain_and_activation(dtype, m, n, k):
    """Every kernel a product can run on: single CTA, split contraction, CTA pairs; stored, and added to an fp32 stream."""
    mo = mops()
    a, w = padded(randn(m, k, seed=1, dtype=dtype)), mo.padded_weight(randn(n, k, seed=2, dtype=dtype, scale=k ** -0.5), dtype, "cuda")
    b, x = randn(n, seed=3), randn(m, n, seed=4)
    r, tol = a.double() @ w.double().t(), 1e-2 if dtype == BF else 3e-5
    close(mo.linear(a, w, bias=b), r + b.double(), tol)
    close(mo.linear(a, w, act="gelu"), O.gelu(r), tol)
    close(mo.linear(a, w, out_dtype=F32, act="cap", cap=1.5, alpha=2.0), O.softcap(2 * r, 1.5), 1e-5 if dtype == BF else 3e-5)
    out = x.clone()
    mo.linear(a, w, out=out, accumulate=True, alpha=0.3, bias=b)
    close(out, x.double() + 0.3 * (r + b.double()), 1e-5 if dtype == BF else 3e-5)
    if n % 8:
        assert torch.equal(mo.linear(a, w, out_dtype=F32), mo.linear(a, w, out_dtype=F32, alpha=1.0))


@pytest.mark.parametrize("dtype", [BF, F32])
def test_grouped_products_with_gelu(dtype):
    mo = mops()
    groups, n, k = dev([2, -1, 0, 2]), 72, 104
    a, w = padded(randn(512, k, seed=1, dtype=dtype)), mo.padded_weight(randn(3 * n, k, seed=2, dtype=dtype, scale=k ** -0.5), dtype, "cuda")
    got = mo.gemm_rows(a, w, groups, n, False, "gelu")
    for t, e in enumerate(groups.tolist()):
        if e >= 0:
            r = a[t * 128:(t + 1) * 128].double() @ w[e * n:(e + 1) * n].double().t()
            close(got[t * 128:(t + 1) * 128], O.gelu(r), 1e-2 if dtype == BF else 1e-5)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("m,heads,k,n", [(1, 3, 24, 7), (130, 20, 128, 128), (300, 5, 40, 72)])
def test_head_products_with_a_gate_per_head_and_steps(dtype, m, heads, k, n):
    mo = mops()
    a, w = padded(randn(m, heads * (k + 8), seed=1, dtype=dtype)), mo.padded_weight(randn(heads * n, k, seed=2, dtype=dtype, scale=k ** -0.5), dtype, "cuda")
    gate = padded(randn(m, heads + 3, seed=3, dtype=dtype))[:, 3:]
    want = torch.stack([a[:, h * (k + 8):h * (k + 8) + k].double() @ w[h * n:(h + 1) * n].double().t() for h in range(heads)], 1)
    tol, step = 1e-2 if dtype == BF else 1e-5, mo.pitch(n) + 8
    out = torch.full((m, heads * step), 7.0, dtype=dtype, device="cuda")
    mo.gemm_heads(a, w, heads, k, n, out=out, a_step=k + 8, c_step=step)
    close(out.view(m, heads, step)[..., :n], want, tol)
    assert (out.view(m, heads, step)[..., n:] == 7.0).all()
    close(mo.gemm_heads(a, w, heads, k, n, gate=gate, a_step=k + 8).reshape(m, heads, n), want * torch.sigmoid(gate.double())[..., None], tol)


# ------------------------------------------------------------------------------------- residual stream and experts
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("d", [5, 44, 320, 2048, 9000])
def test_expert_outputs_join_the_residual_stream(dtype, d):
    mo = mops()
    rows, top = 9, 3
    emb, w = randn(31, d, seed=1, dtype=dtype), randn(d, seed=2, dtype=dtype, scale=0.3)
    y, z, s = (padded(randn(n, d, seed=3 + n, dtype=dtype)) for n in (14, rows, rows))
    tok = dev([0, 30, 4, 4, 9, 1, 2, 3, 30], torch.int64)
    pos = dev([[1, -2, 13], [-1, -1, -1], [0, 2, 3], [-2, -2, -2], [4, 5, 6], [7, 8, 9], [10, -2, 11], [12, -1, 99], [-2, 1, -1]])
    weight, gate = randn(rows, top, seed=9), randn(rows, 5, seed=10)
    x = torch.full((rows, d), float("nan"), device="cuda")
    h, _ = mo.residual_norm(x, w, 1e-3, tokens=tok, embed=emb, embed_scale=2.5, w_offset=1.0)
    close(x, 2.5 * emb[tok].double(), 1e-6)
    tol = 1e-2 if dtype == BF else 5e-6
    close(h, O.centred_norm(x.double(), w.double(), 1e-3), tol)
    add = torch.zeros(rows, d, dtype=torch.float64, device="cuda")
    for r in range(rows):
        for k in range(top):
            p = int(pos[r, k])
            src = y[p] if 0 <= p < 14 else (z[r] if p == -2 else None)
            if src is not None:
                add[r] += weight[r, k].double() * src.double()
    want = x.double() + 0.7 * (add + torch.sigmoid(gate[:, 2:3].double()) * s.double())
    ex = mo.ExpertOutputs(y, pos, 0.7, weight, z, s, gate[:, 2])
    before = x.clone()
    pick, _ = mo.residual_norm(x, w, 1e-3, row_index=dev([8, 0, 6], torch.int64), pending=ex, w_offset=1.0)
    assert torch.equal(x, before)
    close(pick, O.centred_norm(want, w.double(), 1e-3)[[8, 0, 6]], tol)
    h, _ = mo.residual_norm(x, w, 1e-3, pending=ex, w_offset=1.0)
    close(x, want, 5e-6)
    close(h, O.centred_norm(want, w.double(), 1e-3), tol)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows,experts,identity,top,d", [(1, 3, 1, 1, 5), (7, 5, 2, 3, 44), (300, 64, 8, 6, 96), (1500, 4, 0, 4, 40),
                                                            (2000, 300, 3, 9, 72), (129, 1, 1, 2, 64)])
def test_routing_and_dispatch(dtype, rows, experts, identity, top, d):
    """Choices and weights of a router whose scores differ by more than rounding; every chosen expert's rows in its tiles."""
    mo = mops()
    n = experts + identity
    z = torch.stack([torch.linspace(-3, 3, n)[torch.randperm(n, generator=torch.Generator().manual_seed(r))] for r in range(rows)])
    corr = torch.linspace(0.0, 1e-6, n)
    wide = torch.zeros(rows, n + 3, device="cuda")[:, 2:2 + n].copy_(z)
    slots = torch.zeros(rows, dtype=torch.int64, device="cuda")
    slots[3::11] = -1
    live = (slots >= 0).cpu()
    want, wweight = O.route(z.double(), torch.eye(n, dtype=torch.float64), corr.double(), top)
    h = padded(randn(rows, d, seed=3, dtype=dtype))
    for always in (0, 2):                                  # experts that every row uses
        count = torch.zeros(experts, dtype=torch.int32, device="cuda")
        logits = wide if not always else torch.cat((wide, randn(rows, 1, seed=4)), 1)
        choice, rank, weight = mo.moe_route(logits, corr.cuda(), slots, experts, top, count, always)
        assert torch.equal(choice.cpu()[live], want.int()[live]) and (choice.cpu()[~live] == -1).all()
        share = torch.sigmoid(logits[:, n:].double().cpu()).expand(-1, always) if always else torch.zeros(rows, 0, dtype=torch.float64)
        close(weight[live.cuda()], torch.cat((wweight, share), 1)[live], 1e-6)
        dispatched(mo, h, choice, rank, count, live, experts, top, always)


def dispatched(mo, h, choice, rank, count, live, experts, top, always):
    xg, pos, group = mo.moe_dispatch(h, choice, rank, count, always)
    choice, pos, group, count, xg, h = (t.cpu() for t in (choice, pos, group, count, xg, h))
    for a in range(always):
        mine = pos[live, top + a]
        assert (group[(mine // mo.TILE).long()] == experts + a).all() and torch.equal(xg[mine.long()], h[live])
    assert (pos[:, :top][choice >= experts] == -2).all() and (pos[~live] == -1).all()
    pos = pos[:, :top]
    for e in range(experts):
        used = pos[choice == e]
        assert used.unique().numel() == used.numel() == int(count[e]) and (group[(used // mo.TILE).long()] == e).all()
    assert int((group >= 0).sum()) == sum(-(-int(c) // mo.TILE) for c in count) + always * -(-len(h) // mo.TILE)
    r, k = ((choice >= 0) & (choice < experts)).nonzero(as_tuple=True)
    assert torch.equal(xg[pos[r, k].long()], h[r])


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("rows,experts,identity,top,d,always", [(1, 3, 1, 1, 5, 0), (33, 12, 3, 4, 44, 1), (128, 64, 8, 6, 320, 2), (70, 300, 0, 9, 2048, 0)])
def test_few_rows_are_routed_with_the_product(dtype, rows, experts, identity, top, d, always):
    mo = mops()
    n = experts + identity
    h, w = padded(randn(rows, d, seed=1, dtype=dtype)), mo.padded_weight(randn(n + 1, d, seed=2, dtype=dtype, scale=2 * d ** -0.5), dtype, "cuda")
    corr, slots = 0.02 * randn(n, seed=3), torch.zeros(rows, dtype=torch.int64, device="cuda")
    slots[5::7] = -1
    live = (slots >= 0).cpu()
    count, again = torch.zeros(experts, dtype=torch.int32, device="cuda"), torch.zeros(experts, dtype=torch.int32, device="cuda")
    z, choice, rank, weight = mo.moe_route_rows(h, w, corr, slots, experts, top, count, always)
    close(z, h.double() @ w.double().t(), 1e-5)
    c2, _, w2 = mo.moe_route(z[:, :n + (always > 0)], corr, slots, experts, top, again, always)
    assert torch.equal(choice, c2) and torch.equal(count, again) and torch.equal(weight[live.cuda()], w2[live.cuda()])
    dispatched(mo, h, choice, rank, count, live, experts, top, always)


def test_correction_changes_the_choice_but_not_the_weights():
    mo = mops()
    z, corr = dev([[2.0, 1.0, 0.0, -1.0]], F32), dev([-1.0, 0.0, 0.0, 0.9], F32)
    choice, _, weight = mo.moe_route(z, corr, dev([0], torch.int64), 3, 2, torch.zeros(3, dtype=torch.int32, device="cuda"))
    assert choice.tolist() == [[3, 1]]
    close(weight, torch.softmax(torch.tensor([[-1.0, 1.0]]), -1), 1e-6)
    tie, _, _ = mo.moe_route(torch.zeros(1, 70, device="cuda"), torch.zeros(70, device="cuda"), dev([0], torch.int64), 70, 4,
                             torch.zeros(70, dtype=torch.int32, device="cuda"))
    assert tie.tolist() == [[0, 1, 2, 3]]


# ----------------------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,kvr,rot", [(3, 21, 6), (6, 72, 24), (20, 128, 64), (1, 9, 2), (16, 512, 64)])
@pytest.mark.parametrize("absorbed", [0, 3, 7])
def test_rotation_and_append_of_latents(dtype, heads, kvr, rot, absorbed):
    """Every row at its own position; rows whose queries move into latent space beside rows rotated in place; padding rows and other
    slots stay untouched."""
    mo = mops()
    vw, rp = mo.pitch(kvr), mo.pitch(rot)
    width, q_col, kv_col, k_col = vw + rp, 16, 16 + heads * rp, 16 + heads * rp + vw
    proj = padded(randn(7, k_col + rp + 3, seed=1, dtype=dtype))
    wkv, table, rots = randn(kvr, seed=2, dtype=dtype), rotary(100, 300.0, rot), {"base": 300.0, "dims": rot}
    pos, slots = dev([0, 1, 5, 90, 17, 3, 64]), dev([3, 19, -1, 0, 7, 8, 12], torch.int64)
    cache = torch.full((5, 4, width), float("nan"), dtype=dtype, device="cuda")
    ql = torch.full((absorbed, heads * width), 5.0, dtype=dtype, device="cuda") if absorbed else None
    before = proj.clone()
    mo.latent_rotate(proj, q_col, rp, proj, kv_col, k_col, wkv, ql, cache, table, pos, slots, heads, kvr, vw, rot, 1e-4)
    x, tol = before.double().cpu(), 1e-2 if dtype == BF else 1e-5
    q = x[:, q_col:q_col + heads * rp].reshape(7, heads, rp)
    want = O.rotate_interleaved(q[..., :rot], pos.cpu(), rots)
    got = proj[:, q_col:q_col + heads * rp].reshape(7, heads, rp)
    if absorbed < 7:
        close(got[absorbed:, :, :rot], want[absorbed:], tol)
    if absorbed:
        v = ql.view(absorbed, heads, width)
        close(v[..., vw:vw + rot], want[:absorbed], tol)
        assert (v[..., :vw] == 5.0).all() and float(v[..., vw + rot:].abs().sum()) == 0.0
        assert torch.equal(proj[:absorbed], before[:absorbed])
    assert torch.equal(proj[:, :q_col], before[:, :q_col]) and torch.equal(proj[:, kv_col:], before[:, kv_col:])
    flat, live = cache.view(20, -1), slots >= 0
    rows, alive = flat[slots[live]], live.cpu()
    close(rows[:, :kvr], O.rms_norm(x[alive, kv_col:kv_col + kvr], wkv.double().cpu(), 1e-4), tol)
    close(rows[:, vw:vw + rot], O.rotate_interleaved(x[:, None, k_col:k_col + rot], pos.cpu(), rots)[alive, 0], tol)
    assert float(rows[:, kvr:vw].abs().sum()) == 0.0 and float(rows[:, vw + rot:].abs().sum()) == 0.0
    assert int(torch.isnan(flat).any(1).sum()) == 14
    kept = cache.clone()
    mo.latent_rotate(before, q_col, rp, before, None, None, None, ql, cache, table, pos, slots, heads, kvr, vw, rot, 1e-4)      # cache of another layer
    assert torch.equal(cache.nan_to_num(7.0), kept.nan_to_num(7.0))


def latent_case(n, heads, kvr, vw, rot, width, seed, dtype=BF):
    """Cache rows of a sequence, whose keys at the page and tile borders and the first ones may be looked for."""
    c = torch.zeros(n, width)
    g = torch.Generator().manual_seed(seed)
    c[:, :kvr], c[:, vw:vw + rot] = torch.randn(n, kvr, generator=g), torch.randn(n, rot, generator=g)
    return c.to(dtype)


@pytest.mark.parametrize("heads,kvr,rot,page", [(3, 21, 6, 4), (20, 128, 64, 64), (16, 512, 64, 64), (40, 512, 64, 16), (6, 72, 24, 16),
                                                    (33, 256, 32, 128), (8, 256, 8, 8), (17, 384, 56, 32), (5, 300, 64, 64)])
@pytest.mark.parametrize("splits", [0, 1, 3])
def test_latent_decode_with_a_rotated_key_part(heads, kvr, rot, page, splits):
    """One far key per request, found by its rotated part alone, at the first token, at page and tile borders and in the middle."""
    mo = mops()
    vw, width = mo.pitch(kvr), mo.pitch(kvr) + mo.pitch(rot)
    lens = [1, 2, 15, 16, 17, 33, 64, 65, 128, 129, 331]
    far = [0, 0, 3, 15, 16, 0, 63, 63, 64, 127, 128]
    q = torch.zeros(len(lens), heads, width)
    q[..., :kvr], q[..., vw:vw + rot] = torch.randn(len(lens), heads, kvr) * 0.1, torch.randn(len(lens), heads, rot)
    rows = [latent_case(n, heads, kvr, vw, rot, width, n) for n in lens]
    for i in range(len(lens)):
        rows[i][far[i], vw:vw + rot] = (8 * q[i, 0, vw:vw + rot] / q[i, 0, vw:vw + rot].norm()).to(BF)
        q[i, :, vw:vw + rot] = q[i, 0, vw:vw + rot] + 0.2 * q[i, :, vw:vw + rot]
    q = q.to(BF).cuda()
    cache, tables = paged([r.cuda() for r in rows], page)
    pos, slots = dev([n - 1 for n in lens]), torch.zeros(len(lens), dtype=torch.int64, device="cuda")
    slots[4] = -1
    kernels = ["mma", "rows", *(["tcgen05"] if kvr % 128 == 0 and page >= 8 else [])]
    for kernel in kernels:
        got = mo.latent_decode(q.reshape(len(lens), -1), cache, pos, slots, tables, heads, 0, 0.6, splits, kernel, vw)
        for i, n in enumerate(lens):
            if i == 4:
                assert float(got[i].abs().sum()) == 0.0
                continue
            c = rows[i].double()
            s = torch.softmax(q[i].double().cpu() @ c.T * 0.6, -1)
            assert n < 3 or float(s[0, far[i]]) > 0.3
            close(got[i], (s @ c[:, :vw]).reshape(-1), 1.5e-2)


@pytest.mark.parametrize("dtype", [BF, F32])
def test_latent_rows_with_a_rotated_key_part(dtype):
    mo = mops()
    heads, kvr, rot, vw, width, lens = 5, 21, 6, 24, 32, [9, 30]
    rows = [latent_case(n, heads, kvr, vw, rot, width, n, dtype) for n in lens]
    cache, tables = paged([r.cuda() for r in rows], 4)
    q = randn(39, heads * width, seed=3, dtype=dtype)
    seq, pos = dev([0] * 9 + [1] * 30), torch.cat([torch.arange(n) for n in lens]).int().cuda()
    got = mo.latent_attention_rows(q, cache, seq, pos, torch.zeros(39, dtype=torch.int64, device="cuda"), tables, heads, 0, 0.3, vw)
    at = 0
    for i, n in enumerate(lens):
        for t in range(n):
            c = rows[i][:t + 1].double()
            s = torch.softmax(q[at + t].double().cpu().view(heads, width) @ c.T * 0.3, -1)
            close(got[at + t], (s @ c[:, :vw]).reshape(-1), 1e-2 if dtype == BF else 1e-5)
        at += n


@pytest.mark.parametrize("heads,dim,vdim,rot,qp", [(2, 64, 64, 32, 64), (3, 40, 24, 24, 48), (2, 128, 128, 64, 128), (1, 128, 72, 8, 128), (3, 72, 128, 64, 80),
                                                      (2, 16, 104, 6, 16), (2, 128, 40, 16, 128)])
def test_prompt_portions_with_a_rotated_key_part(heads, dim, vdim, rot, qp):
    """Portions of unequal length, some with earlier tokens in front; the last query of each finds one key by the rotated part alone.
    Columns beside a head's own hold other data."""
    mo = mops()
    spans = [(0, 1), (0, 130), (37, 2), (500, 300), (200, 257), (1, 128), (127, 129)]        # (start, tokens)
    vp, rp, kvr = mo.pitch(vdim), mo.pitch(rot), 40
    scale, qs, ks, krs, cu_q, cu_k, want = 1.3 * (dim + rot) ** -0.5, [], [], [], [0], [0], []
    for i, (start, n) in enumerate(spans):
        total = start + n
        g = torch.Generator().manual_seed(i)
        rnd = lambda *sh: torch.randn(*sh, generator=g).to(BF)
        q, qr, k, kr, v = rnd(n, heads, dim), rnd(n, heads, rot), rnd(total, heads, dim), rnd(total, rot), rnd(total, heads, vdim)
        kr[total // 3] = 9 * qr[-1, 0] / qr[-1, 0].float().norm().to(BF)
        s = torch.einsum("nhd,thd->hnt", q.double(), k.double()) + torch.einsum("nhd,td->hnt", qr.double(), kr.double())
        hide = torch.arange(total)[None, :] > torch.arange(start, total)[:, None]
        want.append(torch.einsum("hnt,the->nhe", torch.softmax((s * scale).masked_fill(hide, -math.inf), -1), v.double()).reshape(n, -1))
        pad = lambda t, to: torch.nn.functional.pad(t, (0, to - t.shape[-1])).reshape(len(t), -1)
        qs.append(torch.cat((pad(q, qp), pad(qr, rp), rnd(n, 8)), 1))
        ks.append(torch.cat((pad(k, qp), pad(v, vp)), 1))
        krs.append(torch.cat((rnd(total, kvr), torch.nn.functional.pad(kr, (0, rp - rot))), 1))
        cu_q.append(cu_q[-1] + n)
        cu_k.append(cu_k[-1] + total)
    q, kv, kr = (torch.cat(t).cuda() for t in (qs, ks, krs))
    gates = randn(q.shape[0], heads, seed=5, dtype=BF), padded(randn(q.shape[0], heads * vdim + 3, seed=7, dtype=BF))[:, 3:]
    for gate in (None, *gates):
        out = mo.rows_buffer(q.shape[0], heads * vdim, BF, "cuda")
        mo.window_attention(q, kv, dev(cu_q), dev(cu_k), 300, heads, dim, vdim, 0, scale, out, gate, (qp, qp, vp, heads * qp),
                            (kr, rot, heads * qp, rp, kvr))
        ref = torch.cat(want)
        if gate is not None:
            ref = (ref.view(-1, heads, vdim) * torch.sigmoid(gate.double().cpu()).view(len(ref), heads, -1)).reshape(len(ref), -1)
        close(out, ref, 2e-2)


# ----------------------------------------------------------------------------------------------- grouped attention
def shape(heads, kv, dim, vdim, window, keep=0, cap=0.0, sink=None, rot=0, scale=None, eps=1e-4, whole=True, bias=None):
    sinks = None if sink is None else sink + randn(heads, seed=99)
    return mops().AttentionShape(heads, kv, 1, dim, vdim, rot, 1.5 * dim ** -0.5 if scale is None else scale, window, eps, 0.0, 1.0, bias,
                                 keep, cap, sinks, whole)


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("heads,kv,dim,vdim,rot", [(4, 2, 11, 9, 6), (6, 3, 40, 24, 16), (2, 2, 128, 72, 128), (5, 1, 200, 130, 0), (3, 3, 200, 136, 112),
                                                      (40, 8, 24, 40, 16), (18, 1, 128, 80, 64), (32, 8, 128, 128, 64), (1, 1, 8, 8, 0)])
def test_prepare_norms_over_the_projection(dtype, heads, kv, dim, vdim, rot):
    mo = mops()
    s = shape(heads, kv, dim, vdim, 8, rot=rot)
    rots = {"base": 300.0, "dims": rot, "scaling": {"factor": 3.0}}
    width = (heads + kv) * dim + kv * vdim + 3
    proj = padded(randn(7, width, seed=1, dtype=dtype) * torch.linspace(0.2, 3, width, device="cuda").to(dtype))        # heads of unequal size
    wq, wk = randn(heads * dim, seed=2, dtype=dtype), randn(kv * dim, seed=3, dtype=dtype)
    pos, slots = dev([0, 1, 5, 90, 17, 3, 64]), dev([3, 19, -1, 0, 7, 8, 12], torch.int64)
    cache = torch.full((5, 4, s.cache_width), float("nan"), dtype=dtype, device="cuda")
    table = rotary(100, 300.0, rot, rots["scaling"])
    q = mo.attention_prepare(proj, s, wq, wk, table, pos, slots, cache)
    x, tol = proj.double().cpu(), 1e-2 if dtype == BF else 1e-5
    vectors = lambda cols, n, w: O.rotate_half(O.rms_norm(cols, w.double().cpu(), s.eps).reshape(7, n, dim), pos.cpu(), rots)
    q = q.view(7, heads, s.q_pitch)
    close(q[..., :dim], vectors(x[:, :heads * dim], heads, wq), tol)
    assert float(q[..., dim:].abs().sum()) == 0.0
    flat, live = cache.view(20, -1), slots >= 0
    rows, at = flat[slots[live]], (heads + kv) * dim
    k = rows[:, :kv * s.k_pitch].view(6, kv, s.k_pitch)
    close(k[..., :dim], vectors(x[:, heads * dim:at], kv, wk)[live.cpu()], tol)
    v = rows[:, kv * s.k_pitch:].view(6, kv, s.v_pitch)
    assert torch.equal(v[..., :vdim].reshape(6, -1), proj[live, at:at + kv * vdim])
    assert float(k[..., dim:].abs().sum()) == 0.0 and float(v[..., vdim:].abs().sum()) == 0.0
    assert int(torch.isnan(flat).any(1).sum()) == 14
    before = cache.clone()
    again = mo.attention_prepare(proj, s, wq, None, table, pos, slots, cache)                    # keys of another layer
    assert torch.equal(again.view(7, heads, -1), q) and torch.equal(cache.nan_to_num(7.0), before.nan_to_num(7.0))


def oracle_rows(s, q, k, v):
    cap, sink = s.softcap or 1e9, (torch.full((s.heads,), -1e9) if s.sink is None else s.sink.cpu()).double()
    return O.sink_attention(q.double(), k.double(), v.double(), s.scale, cap, s.window, s.keep, sink)


def case(s, lens, seed=0, dtype=BF, queries=1):
    """Random keys and values of some sequences and the queries of their last ``queries[i]`` positions.  In every sequence four keys agree
    with the last query: the one just inside its window and the last kept one somewhat, the one just outside the window and the
    first that is not kept far more.  -> q, cache rows, expected"""
    g = torch.Generator().manual_seed(seed)
    rnd = lambda *sh: torch.randn(*sh, generator=g).to(dtype)
    qs, rows, want = [], [], []
    for n, nq in zip(lens, queries if isinstance(queries, list) else [queries] * len(lens)):
        q, k, v = rnd(n, s.heads, s.dim), rnd(n, s.kv_heads, s.dim), rnd(n, s.kv_heads, s.vdim)
        a = q[-1, ::s.heads // s.kv_heads].float()
        for at, gain in ((n - s.window, 0.5), (n - 1 - s.window, 1.5), (s.keep - 1, 0.4), (s.keep, 1.2)):
            if 0 <= at < n - 1:
                k[at] = (gain * a / a.norm(dim=-1, keepdim=True) * s.dim ** 0.5).to(dtype)
        want.append(oracle_rows(s, q, k, v)[n - nq:].reshape(nq, -1))
        pad = lambda t, to: torch.nn.functional.pad(t, (0, to - t.shape[-1]))
        qs.append(pad(q[n - nq:], s.q_pitch).reshape(nq, -1))
        rows.append(torch.cat((pad(k, s.k_pitch).reshape(n, -1), pad(v, s.v_pitch).reshape(n, -1)), 1))
    return torch.cat(qs).cuda(), rows, torch.cat(want)


SHAPES = [dict(heads=3, kv=3, dim=24, vdim=40, window=7, keep=3, cap=5.0, sink=1.0), dict(heads=6, kv=2, dim=64, vdim=64, window=44, keep=16, cap=50.0, sink=-1.0),
          dict(heads=12, kv=3, dim=128, vdim=128, window=130, keep=1, cap=20.0, sink=3.0), dict(heads=20, kv=1, dim=40, vdim=72, window=64, keep=17, cap=2.0, sink=0.0),
          dict(heads=4, kv=1, dim=16, vdim=8, window=1, keep=1, cap=10.0, sink=0.5), dict(heads=8, kv=4, dim=104, vdim=128, window=1000, keep=6, cap=8.0, sink=1.0),
          dict(heads=4, kv=2, dim=64, vdim=128, window=33, keep=0, cap=15.0), dict(heads=3, kv=1, dim=24, vdim=24, window=20, keep=150, sink=2.0),
          dict(heads=20, kv=1, dim=128, vdim=96, window=128, keep=128, cap=30.0, sink=1.0), dict(heads=2, kv=2, dim=40, vdim=64, window=65, keep=260, cap=4.0),
          dict(heads=2, kv=1, dim=32, vdim=32, window=16, keep=5), dict(heads=2, kv=1, dim=64, vdim=64, window=40, keep=2, cap=6.0, sink=200.0)]


@pytest.mark.parametrize("kw", SHAPES)
@pytest.mark.parametrize("page", [4, 64])
def test_decode_at_every_edge(kw, page):
    mo, s = mops(), shape(**kw)
    lens = [1, 2, 15, 16, 17, 32, 33, 63, 64, 65, 97, 331]
    q, rows, want = case(s, lens)
    cache, tables = paged([r.cuda() for r in rows], page)
    pos, slots = dev([n - 1 for n in lens]), torch.zeros(len(lens), dtype=torch.int64, device="cuda")
    slots[4] = -1
    live = torch.arange(len(lens)) != 4
    for splits in (0, 1, 3):
        out = torch.zeros(len(lens), s.heads * s.vdim, dtype=BF, device="cuda")
        mo.attention_decode(q, s, cache, pos, slots, tables, out, None, splits)
        close(out[live], want[live], 2e-2)
    mo.attention_rows(q, s, cache, None, pos, slots, tables, out)
    close(out[live], want[live], 1.5e-2)
    assert float(out[4].abs().sum()) == 0.0


@pytest.mark.parametrize("dtype", [BF, F32])
@pytest.mark.parametrize("kw", [dict(heads=4, kv=2, dim=11, vdim=9, window=6, keep=3, cap=3.0, sink=1.0), dict(heads=3, kv=1, dim=150, vdim=140, window=5, keep=9, cap=9.0, sink=0.0),
                                   dict(heads=4, kv=4, dim=10, vdim=12, window=4, keep=2, cap=5.0, sink=-1.0, scale=-0.4)])
def test_general_rows_of_portions(kw, dtype):
    mo, s = mops(), shape(**kw)
    lens = [9, 30]
    q, rows, want = case(s, lens, dtype=dtype, queries=[9, 30])
    cache, tables = paged([r.cuda() for r in rows], 4)
    seq, pos = dev([0] * 9 + [1] * 30), torch.cat([torch.arange(n) for n in lens]).int().cuda()
    out = torch.empty(39, s.heads * s.vdim, dtype=dtype, device="cuda")
    mo.attention_rows(q, s, cache, seq, pos, torch.zeros(39, dtype=torch.int64, device="cuda"), tables, out)
    close(out, want, 1.5e-2 if dtype == BF else 1e-5)


@pytest.mark.parametrize("kw", SHAPES)
@pytest.mark.parametrize("page", [16, 64, 128])
def test_portions_of_prompts(kw, page):
    """Portions of unequal length, some with earlier tokens in front, cut inside tiles and pages."""
    mo, s = mops(), shape(**kw)
    spans = [(0, 1), (0, 130), (37, 2), (300, 290), (200, 57), (1, 128), (127, 129), (600, 3)]        # (start, tokens)
    q, rows, want = case(s, [a + n for a, n in spans], queries=[n for _, n in spans])
    cache, tables = paged([r.cuda() for r in rows], page)
    cu = dev([0, *torch.tensor([n for _, n in spans]).cumsum(0).tolist()])
    pos = torch.cat([torch.arange(a, a + n) for a, n in spans]).int().cuda()
    gate = padded(randn(q.shape[0], s.heads * s.vdim + 3, seed=7, dtype=BF))[:, 3:]
    for g in (None, gate):
        out = mo.rows_buffer(q.shape[0], s.heads * s.vdim, BF, "cuda")
        mo.attention_portions(q, s, cache, pos, cu, 290, tables, out, g)
        close(out, want * (1.0 if g is None else torch.sigmoid(g.double().cpu())), 2e-2)


def test_large_scores_reach_the_cap():
    """Scores far beyond the cap, where its hyperbolic tangent is one."""
    mo, s = mops(), shape(2, 1, 64, 64, 50, keep=3, cap=4.0, sink=1.0, scale=9.0)
    q, rows, want = case(s, [200], queries=[200])
    cache, tables = paged([rows[0].cuda()], 64)
    pos, slots, out = torch.arange(200, dtype=torch.int32, device="cuda"), torch.zeros(200, dtype=torch.int64, device="cuda"), torch.empty(200, 128, dtype=BF, device="cuda")
    mo.attention_portions(q, s, cache, pos, dev([0, 200]), 200, tables, out)
    close(out, want, 2e-2)
    mo.attention_rows(q, s, cache, dev([0] * 200), pos, slots, tables, out)
    close(out, want, 1.5e-2)
    mo.attention_decode(q[-1:].contiguous(), s, cache, pos[-1:], slots[:1], tables, out[:1])
    close(out[:1], want[-1:], 2e-2)


def test_bad_indices_are_reported_not_followed():
    from llm_systems_from_scratch_b200.ops import native
    mo, s = mops(), shape(2, 1, 16, 16, 50, keep=2, cap=5.0, sink=0.0, rot=4)
    proj, w = torch.ones(2, 64, device="cuda", dtype=BF), torch.ones(32, device="cuda", dtype=BF)
    cache, slots, table = torch.zeros(3, 64, 32, device="cuda", dtype=BF), torch.zeros(2, dtype=torch.int64, device="cuda"), rotary(9, 10.0, 4)
    lat = torch.zeros(3, 64, 24, device="cuda", dtype=BF)
    turn = lambda pos, slots: mo.latent_rotate(proj, 0, 8, proj, 16, 32, w[:16], None, lat, table, dev(pos), dev(slots, torch.int64), 2, 16, 16, 4, 1e-4)
    for bad in (lambda: mo.attention_prepare(proj, s, w, w[:16], table, dev([0, 1]), dev([0, 192], torch.int64), cache),
                lambda: mo.attention_prepare(proj, s, w, None, table, dev([0, 9]), slots, cache),
                lambda: turn([0, 1], [0, 192]), lambda: turn([0, 9], [0, 1]),
                lambda: mo.latent_decode(torch.ones(1, 48, device="cuda", dtype=BF), lat, dev([70]), slots[:1], dev([[0, 7]]), 2, 0, 0.3, 1, "mma", 16)):
        bad()
        torch.cuda.synchronize()
        with pytest.raises(native.KernelError):
            native.check_status()


# ------------------------------------------------------------------------------------------- whole models
TOL = {F32: 5e-5, BF: 0.1}            # worst row of a sequence


def agrees(got, want, dtype):
    return H.error(got, want) < TOL[dtype]


def engine(cfg, ts, dtype, **kw):
    from llm_systems_from_scratch_b200.models.genedra import Genedra
    from llm_systems_from_scratch_b200.serving import ServingEngine
    args = dict(num_pages=64, page_size=16, max_batch=4, max_context=512, use_cuda_graphs=False)
    args.update(kw)
    return ServingEngine(Genedra(cfg, ts, dtype, "cuda"), **args)


def weights(cfg, dtype, seed=0):
    """In 16 bits a close call of a router is decided by rounding, so its choices are kept apart there."""
    return H.tensors(cfg, seed, steer=dtype == BF)


@pytest.mark.parametrize("name", list(H.CONFIGS))
@pytest.mark.parametrize("dtype", [F32, BF])
def test_models_in_every_cut_and_company(name, dtype):
    """Whole prompts, token by token, portions down to two tokens, and mixed batches that leave and return, on pages and slots
    that are used again (and poisoned in between), all against the oracle on the whole sequence."""
    cfg = H.CONFIGS[name]
    ts = weights(cfg, dtype)
    seqs = H.prompts(cfg, [170, 33, 1, 64, 90, 130])
    n = [len(s) for s in seqs]
    want = H.expected(cfg, ts, seqs)
    assert dtype == F32 or H.closest_call(cfg, ts, seqs[1:2]) > 0.05
    whole = [[(i, k)] for i, k in enumerate(n)]
    for page in (16, 64):
        eng = engine(cfg, ts, dtype, page_size=page, num_pages=1024 // page)
        for schedule in (whole, sum([H.alone(i, n[i], [n[i] - 40, *[1] * 40] if n[i] > 60 else [1]) for i in range(6)], []),
                         sum([H.alone(i, n[i], [2, 3, 16, 31]) for i in range(6)], []),
                         H.mixed(n, [[50, *[1] * 12], [2], [7, 1, 1], [64, 1], [15, 17, 2, 1]], live=4),
                         [[(0, 100), (1, 33), (3, 64), (4, 90)], [(5, 130), (0, 70), (2, 1)]]):
            got = H.feed(eng, seqs, schedule, poison=True)
            for i in range(6):
                assert agrees(got[i], want[i], dtype), (i, dtype, schedule[:3], H.error(got[i], want[i]))
            assert eng.cache.allocator.free == 1024 // page and eng.cache.slot_allocator.free == 4


def test_residual_stream_after_every_layer():
    from llm_systems_from_scratch_b200.serving.batch import StepBatch
    for name in ("odd", "wide"):
        cfg = H.CONFIGS[name]
        ts = H.tensors(cfg)
        seq = H.prompts(cfg, [50])[0]
        eng = engine(cfg, ts, F32)
        req = eng.open("a")
        eng.sched.grow(req, 50)
        trace = []
        eng.backend.forward(StepBatch.build([(req, 0, seq)], 16, eng.max_pages_per_req, eng.device), trace)
        for a, b in zip(trace, O.Oracle(cfg, ts).residuals(seq)):
            close(a, b, 5e-5)


def test_a_large_batch_decodes_as_each_alone():
    cfg = H.CONFIGS["wide"]
    ts = weights(cfg, BF)
    lens = [5 + (7 * i) % 90 for i in range(70)]
    seqs = H.prompts(cfg, lens)
    eng = engine(cfg, ts, BF, num_pages=160, page_size=64, max_batch=70)
    steps = [[(i, n - 4) for i, n in enumerate(lens)]] + [[(i, 1) for i in range(70)]] * 4
    got = H.feed(eng, seqs, steps, poison=True)
    for i in range(0, 70, 9):
        assert agrees(got[i], H.expected(cfg, ts, [seqs[i]])[0], BF)


@pytest.mark.parametrize("dtype", [F32, BF])
def test_long_decoding_stays_exact(dtype):
    """Past every window, and with kept tokens ever farther away."""
    cfg = H.CONFIGS["tiles"]
    ts = weights(cfg, dtype)
    seq = H.prompts(cfg, [330])
    want = H.expected(cfg, ts, seq)[0]
    got = H.feed(engine(cfg, ts, dtype), seq, H.alone(0, 330, [5, *[1] * 325]))[0]
    assert agrees(got, want, dtype)


@pytest.mark.parametrize("graphs", [False, True])
@pytest.mark.parametrize("dtype", [F32, BF])
def test_greedy_generation_through_the_engine(dtype, graphs):
    """More requests than rows, prompts in portions, captured decode steps; every token is the oracle's choice given the tokens
    before it, unless the two best logits are closer than the precision."""
    cfg = H.CONFIGS["tiles"]
    ts = weights(cfg, dtype)
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
    assert H.error(torch.cat(got), want[[0, 19, 29]]) < 5e-5
