"""Plain, slow statement of the Tedirax design: one function per mechanism, loops where loops are clearest.

Nothing here is shared with the package.  ``Oracle(config, tensors, dtype).logits(tokens)`` runs a whole sequence from
its first token; a decode step, a portion of a prompt or a batch has no counterpart here on purpose - whatever the
framework does with caches and batches has to agree with this.  ``dtype`` is the precision of everything (float64 is
the truth the float32 runs are measured against)."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def rotate_half(x, positions, base, dims):
    """Rotary embedding of (T, heads, dim): dimension i < dims/2 is paired with i + dims/2, the rest stays."""
    if not dims:
        return x
    half = dims // 2
    out = x.clone()
    for i in range(half):
        freq = float(base) ** (-2.0 * i / dims)
        angle = positions.double() * freq
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def retention_scan(q, k, v, decay):
    """q, k (T, H, D), v (T, H, E): S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t, one token at a time."""
    steps, heads, _ = q.shape
    out = torch.zeros(steps, heads, v.shape[-1], dtype=q.dtype)
    decay = torch.as_tensor(decay, dtype=q.dtype)
    state = torch.zeros(heads, q.shape[-1], v.shape[-1], dtype=q.dtype)
    for t in range(steps):
        state = decay[:, None, None] * state + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hde,hd->he", state, q[t])
    return out


def retention(h, w, spec, eps):
    """The whole mixer for one sequence h (T, width); ``w(name)`` gives a weight."""
    steps, heads, dim, vdim = h.shape[0], spec["heads"], spec["dim"], spec["vdim"]
    pos = torch.arange(steps)
    q = (h @ w("q").T).reshape(steps, heads, dim)
    k = (h @ w("k").T).reshape(steps, heads, dim)
    v = (h @ w("v").T).reshape(steps, heads, vdim)
    q = rotate_half(q, pos, spec["rot"]["base"], spec["rot"]["dims"])
    k = rotate_half(k, pos, spec["rot"]["base"], spec["rot"]["dims"]) * dim ** -0.5
    o = rms(retention_scan(q, k, v, spec["decay"]), eps).reshape(steps, heads * vdim)
    g = h @ w("g").T
    return (o * (g * torch.sigmoid(g))) @ w("o").T


def window_attention(q, k, v, scale, size):
    """Softmax attention (T, H, .): position i sees j with 0 <= i - j < size."""
    steps = q.shape[0]
    i = torch.arange(steps)
    seen = (i[:, None] - i[None, :] >= 0) & (i[:, None] - i[None, :] < size)
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    p = torch.softmax(s.masked_fill(~seen, -math.inf), -1)
    return torch.einsum("hij,jhe->ihe", p, v)


def latent_attention(h, w, spec, eps):
    steps, heads, dim, vdim = h.shape[0], spec["heads"], spec["dim"], spec["vdim"]
    cq = rms_norm(h @ w("dq").T, w("dq.norm"), eps)
    c = rms_norm(h @ w("dkv").T, w("dkv.norm"), eps)
    q = (cq @ w("uq").T).reshape(steps, heads, dim)
    k = (c @ w("uk").T).reshape(steps, heads, dim)
    v = (c @ w("uv").T).reshape(steps, heads, vdim)
    o = window_attention(q, k, v, spec["scale"], spec["mask"]["size"]).reshape(steps, heads * vdim)
    return (o * torch.sigmoid(h @ w("g").T)) @ w("o").T


def expert(h, w_gate, w_up, w_down):
    g = h @ w_gate.T
    return ((g * torch.sigmoid(g)) * (h @ w_up.T)) @ w_down.T


def table_moe(h, tokens, table, experts, top):
    """experts: list of (gate, up, down); a token id's row of ``table`` names its ``top`` experts, each with weight 1/top."""
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in table[int(tok)].tolist():
            out[t] += expert(h[t:t + 1], *experts[e])[0] / top
    return out


def layer_order(config):
    n = len(config["layers"])
    loop = config.get("loop")
    if not loop:
        return list(range(n))
    a, b, times = loop["start"], loop["stop"], loop["times"]
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


class Oracle:
    def __init__(self, config, tensors, dtype=torch.float64):
        self.cfg, self.dtype = config, dtype
        self.t = {k: (v if v.dtype == torch.int32 else v.to(dtype)) for k, v in tensors.items()}

    def residuals(self, tokens):
        """The residual stream after every layer run: [layer runs, tokens, width]."""
        cfg, t = self.cfg, self.t
        eps = cfg["norm"]["eps"]
        ids = torch.as_tensor(tokens, dtype=torch.long)
        x = t["embed"][ids]
        out = []
        for i in layer_order(cfg):
            spec, pre = cfg["layers"][i], f"l{i}."
            h = rms_norm(x, t[pre + "norm1"], eps)
            mixer = {"retention": retention, "latent_attention": latent_attention}[spec["type"]]
            y = mixer(h, lambda name: t[pre + "mix." + name], spec["mixer"], eps)
            if spec.get("mlp"):
                n, top = spec["mlp"]["router"]["experts"], spec["mlp"]["router"]["top"]
                ws = [tuple(t[f"{pre}mlp.e{e}.{k}"] for k in ("gate", "up", "down")) for e in range(n)]
                y = y + table_moe(h, ids, t[pre + "mlp.table"], ws, top)
            x = x + y
            out.append(x)
        return torch.stack(out)

    def logits(self, tokens):
        x = self.residuals(tokens)[-1]
        return rms_norm(x, self.t["final.norm"], self.cfg["norm"]["eps"]) @ self.t["head"].T
