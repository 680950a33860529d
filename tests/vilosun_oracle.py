"""Plain, slow statement of the Vilosun design: one function per mechanism, loops where loops are clearest.

Nothing here is shared with the package.  ``Oracle(config, tensors, dtype).logits(tokens)`` runs a whole sequence from
its first token; a decode step, a portion of a prompt or a batch has no counterpart here on purpose - whatever the
framework does with caches and batches has to agree with this.  ``dtype`` is the precision of everything (float64 is
the truth the float32 runs are measured against)."""
from __future__ import annotations

import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def group_norm(x, w, groups, eps):
    """Equal consecutive parts of x, each over its own root mean square; then the weight."""
    parts = x.reshape(*x.shape[:-1], groups, -1)
    return (parts / torch.sqrt((parts * parts).mean(-1, keepdim=True) + eps)).reshape(x.shape) * w


def embed(tokens, table, scale, bigram, spec):
    """Row of the token times the scale, plus the row of (previous token, token); the first token takes the last bigram row."""
    out = []
    for i, t in enumerate(tokens):
        row = spec["buckets"] if i == 0 else (tokens[i - 1] * spec["mul_prev"] + t * spec["mul_cur"]) % spec["buckets"]
        out.append(table[t] * scale + bigram[row])
    return torch.stack(out)


def short_conv(u, w):
    """y_t = sum_j w[:, j] u_(t - taps + 1 + j) per channel, zeros in front of the sequence.  u (T, channels), w (channels, taps)."""
    taps, y = w.shape[1], torch.zeros_like(u)
    for t in range(len(u)):
        for j in range(taps):
            if t - taps + 1 + j >= 0:
                y[t] += w[:, j] * u[t - taps + 1 + j]
    return y


# ------------------------------------------------------------------------------------------------- attention
def visible(i, j, size):
    return j <= i and i // size == j // size


def slope(h, heads):
    return 2.0 ** (-8.0 * (h + 1) / heads)


def chunked_attention(q, k, v, scale, temp, size):
    """q (T, H, D), k (T, G, D), v (T, G, E): scores times a number per head, less slope times distance, inside the position's chunk."""
    steps, heads = q.shape[0], q.shape[1]
    rep = heads // k.shape[1]
    mask = torch.tensor([[visible(i, j, size) for j in range(steps)] for i in range(steps)])
    at = torch.arange(steps, dtype=q.dtype)
    out = torch.zeros(steps, heads, v.shape[-1], dtype=q.dtype)
    for h in range(heads):
        s = q[:, h] @ k[:, h // rep].T * scale * temp[h] - slope(h, heads) * (at[:, None] - at[None])
        out[:, h] = torch.softmax(s.masked_fill(~mask, -math.inf), -1) @ v[:, h // rep]
    return out


def attention(h, w, spec, v_first):
    """Returns the mixer's output and its (mixed) values (T, G * E)."""
    steps, heads, kv, dim = len(h), spec["heads"], spec["kv_heads"], spec["dim"]
    proj = lambda name: short_conv(h @ w(name).T + w(name + ".b"), w(name + ".conv"))
    q, k, v = proj("q").reshape(steps, heads, dim), proj("k").reshape(steps, kv, dim), proj("v")
    if v_first is not None:
        v = (1 - w("vmix")) * v + w("vmix") * v_first
    o = chunked_attention(q, k, v.reshape(steps, kv, -1), spec["scale"], w("temp"), spec["mask"]["size"])
    return (o * sigmoid(h @ w("g").T)[..., None]).reshape(steps, -1) @ w("o").T, v


# ------------------------------------------------------------------------------------------------ delta rule
def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, g, beta):
    """q, k (T, H, D), v (T, H, E), decay g and write strength beta (T, H): decay, correct what is stored at k, read."""
    steps, heads, dim = q.shape
    out = torch.zeros_like(v)
    for h in range(heads):
        S = torch.zeros(dim, v.shape[-1], dtype=q.dtype)
        for t in range(steps):
            S = g[t, h] * S
            u = beta[t, h] * (v[t, h] - S.T @ k[t, h])
            S = S + torch.outer(k[t, h], u)
            out[t, h] = S.T @ q[t, h]
    return out


def log_decay(h, w):
    z = h @ w("a").T + w("dt_bias")
    return -torch.exp(w("A_log")) * torch.where(z > 30, z, torch.log1p(torch.exp(z.clamp(max=30))))


def delta(h, w, spec, eps):
    steps, heads, kv, dim, vdim = len(h), spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    proj = lambda name: silu(short_conv(h @ w(name).T, w(name + ".conv")))
    rep = lambda x: x.reshape(steps, kv, dim).repeat_interleave(heads // kv, 1)
    q, k = rep(unit(proj("q").reshape(steps, kv, dim))) * dim ** -0.5, rep(unit(proj("k").reshape(steps, kv, dim)))
    o = delta_rule(q, k, proj("v").reshape(steps, heads, vdim), torch.exp(log_decay(h, w)), sigmoid(h @ w("b").T))
    o = o / torch.sqrt((o * o).mean(-1, keepdim=True) + eps) * w("norm")
    return (o.reshape(steps, -1) * silu(h @ w("g").T)) @ w("o").T


# ---------------------------------------------------------------------------------------------- feed-forward
def expert(h, w_gate, w_up, w_down):
    return (silu(h @ w_gate.T) * (h @ w_up.T)) @ w_down.T


def route(z, top):
    """The largest logits and the softmax over them."""
    best = torch.topk(z, top, dim=-1)
    return best.indices, torch.softmax(best.values, -1)


def mixture(h, w, spec):
    chosen, weight = route(h @ w("router").T + w("router.b"), spec["router"]["top"])
    out = torch.zeros_like(h)
    for t in range(len(h)):
        for e, a in zip(chosen[t].tolist(), weight[t]):
            out[t] += a * expert(h[t:t + 1], w(f"e{e}.gate"), w(f"e{e}.up"), w(f"e{e}.down"))[0]
    return out


class Oracle:
    def __init__(self, config, tensors, dtype=torch.float64):
        self.cfg, self.dtype = config, dtype
        self.t = {k: v.to(dtype) for k, v in tensors.items()}

    def residuals(self, tokens):
        """The residual stream after every layer: [layers, tokens, width]."""
        cfg, t = self.cfg, self.t
        eps, groups = cfg["norm"]["eps"], cfg["norm"]["groups"]
        x = embed([int(i) for i in tokens], t["embed"], cfg["embedding"]["scale"], t["bigram"], cfg["embedding"]["bigram"])
        out, v_first = [], None

        def sublayer(x, pre, n, run):
            h = group_norm(x, t[f"{pre}norm{n}"], groups, eps)
            y = run(h) * sigmoid(h @ t[f"{pre}rg{n}"].T + t[f"{pre}rg{n}.b"])
            return x + group_norm(y, t[f"{pre}norm{n}b"], groups, eps)
        for i, layer in enumerate(cfg["layers"]):
            pre, spec = f"l{i}.", layer["mixer"]
            w = lambda name: t[pre + "mix." + name]
            if layer["type"] == "attention":
                kept = []

                def run(h):
                    y, v = attention(h, w, spec, v_first if spec["v_mix"] else None)
                    kept.append(v)
                    return y
                x = sublayer(x, pre, 1, run)
                if spec["v_mix"] and v_first is None:
                    v_first = kept[0]
            else:
                x = sublayer(x, pre, 1, lambda h: delta(h, w, spec, eps))
            if layer.get("mlp"):
                w2 = lambda name: t[pre + "mlp." + name]
                x = sublayer(x, pre, 2, lambda h: mixture(h, w2, layer["mlp"]))
            out.append(x)
        return torch.stack(out)

    def logits(self, tokens):
        x = self.residuals(tokens)[-1]
        return group_norm(x, self.t["final.norm"], self.cfg["norm"]["groups"], self.cfg["norm"]["eps"]) @ self.t["head"].T * self.cfg["logit_scale"]
