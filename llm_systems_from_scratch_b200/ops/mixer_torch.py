"""PyTorch statements of the ops behind the layered decoders (``ops.mixer_ops``): what each kernel computes, in fp32, on
CPU tensors.  They let the engine, the cache manager and the scheduler run without a GPU; on a GPU the kernels run."""
from __future__ import annotations

import torch

TILE = 128


def residual_norm(x, tokens, embed, row_index, pending, w, eps, scatter):
    src = x if tokens is None else embed[tokens.long()].float()
    if row_index is not None:
        src = x[row_index.long()]
    if pending is not None:
        y, pos, scale = pending
        rows = pos if row_index is None else pos[row_index.long()]
        live = rows >= 0
        src = src + scale * (y.float()[rows.clamp(min=0).long()] * live.unsqueeze(-1)).sum(1)
    if row_index is None:
        x.copy_(src)
    if w is None:
        return None, None
    h = (src * torch.rsqrt(src.pow(2).mean(-1, keepdim=True) + eps) * w.float()).to(w.dtype)
    if scatter is None:
        return h, None
    pos, rows = scatter
    xg = torch.zeros((rows, x.shape[1]), dtype=h.dtype)
    for k in range(pos.shape[1]):
        live = pos[:, k] >= 0
        xg[pos[live, k].long()] = h[live]
    return h, xg


def moe_plan(tokens, slots, tables, experts, tiles):
    pos, groups = [], []
    for table, n in zip(tables, experts):
        top = table.shape[1]
        where = torch.full((tokens.numel(), top), -1, dtype=torch.int32)
        tile = torch.full((tiles,), -1, dtype=torch.int32)
        at = 0
        chosen = table[tokens.long()]
        chosen = torch.where((slots < 0).unsqueeze(1), torch.full_like(chosen, -1), chosen)
        for e in range(n):
            hit = (chosen == e).nonzero()
            if len(hit):
                where[hit[:, 0], hit[:, 1]] = torch.arange(len(hit), dtype=torch.int32) + at * TILE
                used = -(-len(hit) // TILE)
                tile[at:at + used] = e
                at += used
        pos.append(where)
        groups.append(tile)
    return pos, groups


def gemm_rows(a, w, tile_group, group_rows, n, swiglu):
    out = torch.zeros((a.shape[0], n), dtype=a.dtype)
    for t, e in enumerate(tile_group.tolist()):
        if e < 0:
            continue
        r = a[t * TILE:(t + 1) * TILE].float() @ w[e * group_rows:(e + 1) * group_rows].float().t()
        if swiglu:
            r = torch.nn.functional.silu(r[:, :n]) * r[:, n:]
        out[t * TILE:(t + 1) * TILE] = r.to(a.dtype)
    return out


def gemm_heads(a, w, heads, k, n, out, gate):
    group = w.shape[0] // heads
    for h in range(heads):
        r = a[:, h * k:(h + 1) * k].float() @ w[h * group:h * group + n, :k].float().t()
        if gate is not None:
            r = r * torch.sigmoid(gate[:, h * n:(h + 1) * n].float())
        out[:, h * n:(h + 1) * n] = r.to(out.dtype)
    return out


def latent_norm_append(proj, wq, wkv, eps, cache, slots, cq):
    qr, kvr = wq.numel(), wkv.numel()
    norm = lambda t, w: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    cq.copy_(norm(proj[:, :qr].float(), wq).to(cq.dtype))
    live = slots >= 0
    flat = cache.view(-1, cache.shape[-1])
    flat[slots[live], :kvr] = norm(proj[live, qr:qr + kvr].float(), wkv).to(cache.dtype)
    return cq


def latent_attention(q, cache, row_seq, positions, slots, tables, heads, window, scale):
    width, page = cache.shape[-1], cache.shape[1]
    out = torch.zeros_like(q)
    flat = cache.view(-1, width)
    for r in range(q.shape[0]):
        if slots[r] < 0:
            continue
        p = int(positions[r])
        j = torch.arange(max(0, p - window + 1) if window > 0 else 0, p + 1)
        line = tables[int(row_seq[r]) if row_seq is not None else r].long()
        c = flat[line[j // page] * page + j % page].float()
        s = torch.einsum("hw,jw->hj", q[r].float().view(heads, width), c) * scale
        out[r] = torch.einsum("hj,jw->hw", torch.softmax(s, -1), c).reshape(-1).to(q.dtype)
    return out


def retention(proj, state, state_slots, spans, positions, cos_sin, decay, heads, dim, vdim, rot, eps, y):
    """``spans``: (first row, one past the last row) of every sequence."""
    qkv = proj.float()
    hd, he, half = heads * dim, heads * vdim, rot // 2
    for s, (a, b) in enumerate(spans):
        slot = int(state_slots[s])
        if slot < 0:
            y[a:b] = 0
            continue
        for r in range(a, b):
            pos = int(positions[r])
            S = state[slot]
            if pos == 0:
                S.zero_()

            def rotated(t):
                t = t.clone()
                if rot:
                    c, sn = cos_sin[0, pos], cos_sin[1, pos]
                    u, v = t[:, :half].clone(), t[:, half:rot].clone()
                    t[:, :half], t[:, half:rot] = u * c - v * sn, v * c + u * sn
                return t
            q = rotated(qkv[r, :hd].view(heads, dim))
            k = rotated(qkv[r, hd:2 * hd].view(heads, dim)) * dim ** -0.5
            v = qkv[r, 2 * hd:2 * hd + he].view(heads, vdim)
            S.mul_(decay.view(-1, 1, 1)).add_(k.unsqueeze(2) * v.unsqueeze(1))
            o = torch.einsum("hde,hd->he", S, q)
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
            g = qkv[r, 2 * hd + he:2 * hd + 2 * he].view(heads, vdim)
            y[r] = (o * torch.nn.functional.silu(g)).reshape(-1).to(y.dtype)
    return y
