"""PyTorch statements of the ops behind the layered decoders (``ops.mixer_ops``): what each kernel computes, in fp32, on
CPU tensors.  They let the engine, the cache manager and the scheduler run without a GPU; on a GPU the kernels run."""
from __future__ import annotations

import torch

TILE = 128


def finish(r, bias, alpha, act, cap):
    r = alpha * (r if bias is None else r + bias)
    if act == "gelu":
        return torch.nn.functional.gelu(r)
    return cap * torch.tanh(r / cap) if act == "cap" else r


def residual_norm(x, tokens, embed, row_index, pending, w, eps, scatter, embed_scale, w_offset):
    src = x if tokens is None else embed[tokens.long()].float() * embed_scale
    pick = (lambda t: t) if row_index is None else (lambda t: t[row_index.long()])
    if row_index is not None:
        src = x[row_index.long()]
    if pending is not None:
        rows = pick(pending.pos)
        weight = (rows >= 0).float() if pending.weight is None else pick(pending.weight)
        part = pending.y.float()[rows.clamp(min=0).long()].masked_fill((rows < 0).unsqueeze(-1), 0.0)
        if pending.z is not None:
            part = torch.where((rows == -2).unsqueeze(-1), pick(pending.z).float().unsqueeze(1), part)
        total = (part * weight.unsqueeze(-1)).sum(1)
        if pending.s is not None:
            share = 1.0 if pending.sgate is None else torch.sigmoid(pick(pending.sgate)).unsqueeze(1)
            total = total + share * pick(pending.s).float()
        src = src + pending.scale * total
    if row_index is None:
        x.copy_(src)
    if w is None:
        return None, None
    h = (src * torch.rsqrt(src.pow(2).mean(-1, keepdim=True) + eps) * (w.float() + w_offset)).to(w.dtype)
    if scatter is None:
        return h, None
    pos, rows = scatter
    xg = torch.zeros((rows, x.shape[1]), dtype=h.dtype)
    for k in range(pos.shape[1]):
        live = pos[:, k] >= 0
        xg[pos[live, k].long()] = h[live]
    return h, xg


def add_normed(x, y, w, eps, tokens, embed, h):
    if tokens is not None:
        x.copy_(embed[tokens.long()].float())
    else:
        f = y.float()
        x.add_(f * torch.rsqrt(f.pow(2).mean(-1, keepdim=True) + eps) * w.float())
    return h.copy_(x)


def glu(a, w, n, act, out):
    g, u = (a.float() @ w.float().t()).split(n, 1)
    return out.copy_((torch.relu(g) if act == "relu" else torch.nn.functional.silu(g)) * u)


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


def moe_route(z, correction, slots, experts, top, count, always, bias):
    outputs = z.shape[1] - (always > 0)
    logits = z[:, :outputs] if bias is None else z[:, :outputs] + bias
    s = torch.softmax(logits, -1)
    choice = torch.topk(logits if correction is None else s + correction, top, dim=-1).indices
    weight = s.gather(1, choice)
    weight = weight / (weight.sum(-1, keepdim=True) + 1e-20)
    if always:
        weight = torch.cat((weight, torch.sigmoid(z[:, outputs:]).expand(-1, always)), 1)
    choice, rank = choice.to(torch.int32), torch.full(choice.shape, -1, dtype=torch.int32)
    choice[slots < 0], weight[slots < 0] = -1, 0.0
    for r in range(z.shape[0]):
        for k, e in enumerate(choice[r].tolist()):
            if 0 <= e < experts:
                rank[r, k] = count[e]
                count[e] += 1
    return choice, rank, weight


def moe_dispatch(h, choice, rank, count, always, tiles):
    rows, experts = len(h), count.numel()
    used = -(-torch.cat((count, torch.full((always,), rows, dtype=count.dtype))) // TILE)
    start = torch.cumsum(used, 0) - used
    group = torch.full((tiles,), -1, dtype=torch.int32)
    for e, n in enumerate(used.tolist()):
        group[int(start[e]):int(start[e]) + n] = e
    known = (choice >= 0) & (choice < experts)
    pos = torch.where(known, start[choice.clamp(0, experts - 1).long()].to(torch.int32) * TILE + rank, -1).to(torch.int32)
    pos[choice >= experts] = -2
    more = torch.arange(rows)[:, None] + start[None, experts:] * TILE
    pos = torch.cat((pos, torch.where(choice[:, :1] >= 0, more, -1).to(torch.int32)), 1)
    xg = torch.zeros((tiles * TILE, h.shape[1]), dtype=h.dtype)
    for k in range(pos.shape[1]):
        live = pos[:, k] >= 0
        xg[pos[live, k].long()] = h[live]
    return xg, pos, group


def gemm_rows(a, w, tile_group, group_rows, n, swiglu, act):
    out = torch.zeros((a.shape[0], n), dtype=a.dtype)
    for t, e in enumerate(tile_group.tolist()):
        if e < 0:
            continue
        r = a[t * TILE:(t + 1) * TILE].float() @ w[e * group_rows:(e + 1) * group_rows].float().t()
        if swiglu:
            r = torch.nn.functional.silu(r[:, :n]) * r[:, n:]
        r = finish(r, None, 1.0, act, 0.0)
        out[t * TILE:(t + 1) * TILE] = r.to(a.dtype)
    return out


def gemm_heads(a, w, heads, k, n, out, gate, a_step, c_step):
    group = w.shape[0] // heads
    for h in range(heads):
        r = a[:, h * a_step:h * a_step + k].float() @ w[h * group:h * group + n, :k].float().t()
        if gate is not None:
            g = gate[:, h:h + 1] if gate.shape[1] == heads else gate[:, h * n:(h + 1) * n]
            r = r * torch.sigmoid(g.float())
        out[:, h * c_step:h * c_step + n] = r.to(out.dtype)
    return out


def latent_rotate(proj, q_col, q_pitch, kv, kv_col, k_col, wkv, ql, cache, cos_sin, positions, slots, heads, kv_rank, vwidth, rot, eps):
    c, sn = cos_sin[0, positions.long()], cos_sin[1, positions.long()]

    def turned(t):                                   # (R, ..., rot): pairs (2i, 2i + 1)
        shape = (-1, *[1] * (t.dim() - 2), rot // 2)
        u, v, cc, ss = t[..., 0::2].float(), t[..., 1::2].float(), c.view(shape), sn.view(shape)
        return torch.stack((u * cc - v * ss, v * cc + u * ss), -1).flatten(-2)
    live, n, width = slots >= 0, 0 if ql is None else ql.shape[0], cache.shape[-1]
    flat = cache.view(-1, width)
    if k_col is not None:
        flat[slots[live], vwidth:] = 0
        flat[slots[live], vwidth:vwidth + rot] = turned(kv[:, k_col:k_col + rot])[live].to(cache.dtype)
    if kv_col is not None:
        t = kv[live, kv_col:kv_col + kv_rank].float()
        flat[slots[live], kv_rank:vwidth] = 0
        flat[slots[live], :kv_rank] = (t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * wkv.float()).to(cache.dtype)
    parts = turned(torch.stack([proj[:, q_col + h * q_pitch:q_col + h * q_pitch + rot] for h in range(heads)], 1)).to(proj.dtype)
    if n:
        ql.view(n, heads, width)[..., vwidth:] = 0
        ql.view(n, heads, width)[..., vwidth:vwidth + rot] = parts[:n]
    for h in range(heads):
        proj[n:, q_col + h * q_pitch:q_col + h * q_pitch + rot] = parts[n:, h]


def latent_norm_append(proj, wq, wkv, eps, cache, slots, cq):
    qr, kvr = wq.numel(), wkv.numel()
    norm = lambda t, w: t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + eps) * w.float()
    cq.copy_(norm(proj[:, :qr].float(), wq).to(cq.dtype))
    live = slots >= 0
    flat = cache.view(-1, cache.shape[-1])
    flat[slots[live], :kvr] = norm(proj[live, qr:qr + kvr].float(), wkv).to(cache.dtype)
    return cq


def latent_attention(q, cache, row_seq, positions, slots, tables, heads, window, scale, vwidth):
    width, page = cache.shape[-1], cache.shape[1]
    out = torch.zeros((q.shape[0], heads * vwidth), dtype=q.dtype)
    flat = cache.view(-1, width)
    for r in range(q.shape[0]):
        if slots[r] < 0:
            continue
        p = int(positions[r])
        j = torch.arange(max(0, p - window + 1) if window > 0 else 0, p + 1)
        line = tables[int(row_seq[r]) if row_seq is not None else r].long()
        c = flat[line[j // page] * page + j % page].float()
        s = torch.einsum("hw,jw->hj", q[r].float().view(heads, width), c) * scale
        out[r] = torch.einsum("hj,jw->hw", torch.softmax(s, -1), c[:, :vwidth]).reshape(-1).to(q.dtype)
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


def mlstm(proj, gates, gate_bias, weight, state, state_slots, spans, positions, heads, dim, vdim, cap, eps, y):
    """``spans``: (first row, one past the last row) of every sequence."""
    rows, hd, he = proj.float(), heads * dim, heads * vdim
    logs = cap * torch.tanh((gates + gate_bias) / cap)
    for s, (a, b) in enumerate(spans):
        slot = int(state_slots[s])
        if slot < 0:
            y[a:b] = 0
            continue
        flat = state[slot]
        S, N, M = flat[:, :dim * vdim].view(heads, dim, vdim), flat[:, dim * vdim:dim * vdim + dim], flat[:, dim * vdim + dim]
        for r in range(a, b):
            if int(positions[r]) == 0:
                flat.zero_()
            q, k = rows[r, :hd].view(heads, dim) * dim ** -0.5, rows[r, hd:2 * hd].view(heads, dim)
            v, g = rows[r, 2 * hd:2 * hd + he].view(heads, vdim), rows[r, 2 * hd + he:2 * hd + 2 * he]
            i, f = logs[r, :heads], torch.nn.functional.logsigmoid(logs[r, heads:])
            m = torch.maximum(f + M, i)
            keep, take = torch.exp(f + M - m), torch.exp(i - m)
            M.copy_(m)
            kt = take[:, None] * k
            S.mul_(keep[:, None, None]).add_(kt[:, :, None] * v[:, None, :])
            N.mul_(keep[:, None]).add_(kt)
            o = torch.einsum("hde,hd->he", S, q) / (torch.maximum((N * q).sum(-1).abs(), torch.exp(-m)) + 1e-6)[:, None]
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)
            y[r] = (o.reshape(-1) * weight.float() * torch.sigmoid(g)).to(y.dtype)
    return y


def attention_prepare(proj, s, wq, wk, cos_sin, positions, slots, cache, q):
    half = s.rot // 2

    def vectors(cols, n, w):
        t = cols.float() if s.whole_norm else cols.float().reshape(-1, n, s.dim)
        t = (t * torch.rsqrt(t.pow(2).mean(-1, keepdim=True) + s.eps) * w.float()).reshape(-1, n, s.dim)
        if half:
            c, sn = cos_sin[0, positions.long()][:, None], cos_sin[1, positions.long()][:, None]
            u, v = t[..., :half], t[..., half:s.rot]
            t = torch.cat((u * c - v * sn, v * c + u * sn, t[..., s.rot:]), -1)
        return t
    nq, nk = s.heads * s.maps, s.kv_heads * s.maps
    q.zero_().view(-1, nq, s.q_pitch)[..., :s.dim] = vectors(proj[:, :nq * s.dim], nq, wq).to(q.dtype)
    if wk is not None:
        live, at = slots >= 0, (nq + nk) * s.dim
        row = torch.zeros((proj.shape[0], s.cache_width), dtype=cache.dtype)
        row[:, :nk * s.k_pitch].view(-1, nk, s.k_pitch)[..., :s.dim] = vectors(proj[:, nq * s.dim:at], nk, wk).to(cache.dtype)
        row[:, nk * s.k_pitch:].view(-1, s.kv_heads, s.v_pitch)[..., :s.vdim] = proj[:, at:at + s.kv_heads * s.vdim].view(-1, s.kv_heads, s.vdim)
        cache.view(-1, s.cache_width)[slots[live]] = row[live]
    return q


def attention_rows(q, s, cache, row_seq, positions, slots, tables, out, gate):
    page, flat = cache.shape[1], cache.view(-1, s.cache_width)
    keys = s.kv_heads * s.maps * s.k_pitch
    rep = s.heads // s.kv_heads
    for r in range(q.shape[0]):
        if slots[r] < 0:
            out[r] = 0
            continue
        p = int(positions[r])
        lo = p - p % s.window if s.chunked else max(0, p - s.window + 1)
        j = torch.cat((torch.arange(min(s.keep, lo)), torch.arange(lo, p + 1)))
        line = tables[int(row_seq[r]) if row_seq is not None else r].long()
        c = flat[line[j // page] * page + j % page].float()
        k = c[:, :keys].view(-1, s.kv_heads, s.maps, s.k_pitch)[..., :s.dim].repeat_interleave(rep, 1)
        v = c[:, keys:].view(-1, s.kv_heads, s.v_pitch)[..., :s.vdim].repeat_interleave(rep, 1)
        score = torch.einsum("hmd,jhmd->hmj", q[r].float().view(s.heads, s.maps, s.q_pitch)[..., :s.dim], k) * s.scale
        if s.softcap:
            score = s.softcap * torch.tanh(score / s.softcap)
        if s.bias is not None:
            score = score + s.bias[:, (p - j).clamp(max=s.bias.shape[1] - 1)][:, None]
        if s.slopes is not None:
            score = score - (s.slopes[:, None] * (p - j))[:, None]
        if s.sink is not None:
            score = torch.cat((score, s.sink.view(-1, 1, 1).expand(-1, s.maps, 1)), -1)
        o = torch.einsum("hmj,jhe->hme", torch.softmax(score, -1)[..., :len(j)], v)
        if s.maps == 2:
            o = o[:, 0] - s.difference * o[:, 1]
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + s.eps) * s.out_scale
        o = o.reshape(-1)
        if gate is not None:
            o = o * torch.sigmoid(gate[r].float()).repeat_interleave(len(o) // gate.shape[1])
        out[r] = o.to(out.dtype)
    return out


def short_conv(u, w, ring, at, silu):
    taps, f, y = w.shape[0], u.float(), torch.zeros_like(u, dtype=torch.float32)
    kept = ring.clone()
    for seq, (a, b) in enumerate(at.spans):
        slot = int(at.state_slots[seq])
        for r in range(a, b):
            pos = int(at.positions[r])
            for d in range(taps):
                if r - d >= a:
                    y[r] += w[taps - 1 - d].float() * f[r - d]
                elif pos >= d and slot >= 0:
                    y[r] += w[taps - 1 - d].float() * kept[slot, (pos - d) % taps].float()
            if slot >= 0:
                ring[slot, pos % taps] = u[r]
    return torch.nn.functional.silu(y).to(u.dtype) if silu else y.to(u.dtype)


def conv_attend(u, w, ring, at, s, temp, cache, first, mix, q):
    c = short_conv(u.float(), w.float(), ring, at, False)
    nq, nk = s.heads * s.dim, s.kv_heads * s.dim
    q.zero_().view(-1, s.heads, s.q_pitch)[..., :s.dim] = c[:, :nq].view(-1, s.heads, s.dim) * temp[:, None]
    live = at.slots >= 0
    v = c[:, nq + nk:].view(-1, s.kv_heads, s.vdim)
    if first is not None:
        vf = first.view(-1, first.shape[-1])[at.slots.clamp(min=0)][:, first.shape[-1] - s.kv_heads * s.v_pitch:]
        v = (1.0 - mix) * v + mix * vf.reshape(-1, s.kv_heads, s.v_pitch)[..., :s.vdim].float()
    row = torch.zeros((len(u), s.cache_width), dtype=cache.dtype)
    row[:, :s.kv_heads * s.k_pitch].view(-1, s.kv_heads, s.k_pitch)[..., :s.dim] = c[:, nq:nq + nk].view(-1, s.kv_heads, s.dim).to(cache.dtype)
    row[:, s.kv_heads * s.k_pitch:].view(-1, s.kv_heads, s.v_pitch)[..., :s.vdim] = v.to(cache.dtype)
    cache.view(-1, s.cache_width)[at.slots[live]] = row[live]
    return q


def delta_rule(c, gate, ab, decay, dt, weight, state, at, kv_heads, eps, y):
    _, heads, dim, vdim = state.shape
    rep = lambda t: t.view(kv_heads, dim).repeat_interleave(heads // kv_heads, 0)
    unit = lambda t: t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + 1e-6)
    g, beta = torch.exp(decay * torch.nn.functional.softplus(ab[:, :heads] + dt)), torch.sigmoid(ab[:, heads:])
    for seq, (a, b) in enumerate(at.spans):
        slot = int(at.state_slots[seq])
        if slot < 0:
            y[a:b] = 0
            continue
        S = state[slot]
        for r in range(a, b):
            if int(at.positions[r]) == 0:
                S.zero_()
            row = c[r].float()
            q, k = unit(rep(row[:kv_heads * dim])) * dim ** -0.5, unit(rep(row[kv_heads * dim:2 * kv_heads * dim]))
            S.mul_(g[r][:, None, None])
            u = beta[r][:, None] * (row[2 * kv_heads * dim:].view(heads, vdim) - torch.einsum("hde,hd->he", S, k))
            S.add_(k[:, :, None] * u[:, None])
            o = torch.einsum("hde,hd->he", S, q)
            o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps) * weight.float()
            y[r] = (o.reshape(-1) * torch.nn.functional.silu(gate[r].float())).to(y.dtype)
    return y


def group_step(x, groups, eps, w, start, batch, sub, row_index):
    def norm(t, weight):
        parts = t.view(len(t), groups, -1)
        return (parts * torch.rsqrt(parts.pow(2).mean(-1, keepdim=True) + eps)).view(t.shape) * weight.float()
    pick = (lambda t: t) if row_index is None else (lambda t: t[row_index.long()])
    src = pick(x)
    if start is not None:
        src = start.embed[batch.tokens].float() * start.scale
        if start.bigram is not None:
            buckets, seen = len(start.bigram) - 1, {}
            for r in range(len(x)):
                seq, tok = int(batch.row_seq[r]), int(batch.tokens[r])
                slot = int(batch.state_slots[seq])
                before = seen.get(seq, int(start.prev[slot]) if slot >= 0 else 0)
                pair = buckets if int(batch.positions[r]) == 0 else (before * start.mul_prev + tok * start.mul_cur) % buckets
                src[r] += start.bigram[pair].float()
                seen[seq] = tok
                if slot >= 0:
                    start.prev[slot] = tok
    if sub is not None:
        if isinstance(sub.y, torch.Tensor):
            u = pick(sub.y).float()
        else:
            pos = pick(sub.y.pos)
            part = sub.y.y.float()[pos.clamp(min=0).long()].masked_fill((pos < 0).unsqueeze(-1), 0.0)
            u = (part * pick(sub.y.weight).unsqueeze(-1)).sum(1)
        src = src + norm(u * torch.sigmoid(pick(sub.gate).float()), sub.w_post)
    if row_index is None:
        x.copy_(src)
    return None if w is None else norm(src, w).to(w.dtype)
