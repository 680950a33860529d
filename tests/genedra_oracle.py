"""Plain, slow statement of the Genedra design: one function per mechanism, loops where loops are clearest.

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


def centred_norm(x, w, eps):
    """The weight is stored as its distance from one."""
    return rms(x, eps) * (1 + w)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


# -------------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    factor = (rot.get("scaling") or {"factor": 1.0})["factor"]
    return [float(rot["base"]) ** (-2.0 * i / rot["dims"]) / factor for i in range(rot["dims"] // 2)]


def turn(x, positions, rot, pairs):
    """Turn the pairs (a, b) of dimensions of x (T, heads, dim) by position * frequency; the others stay."""
    out = x.clone()
    for f, (a, b) in zip(frequencies(rot), pairs):
        angle = positions.double() * f
        c, s = torch.cos(angle).to(x.dtype)[:, None], torch.sin(angle).to(x.dtype)[:, None]
        out[..., a] = x[..., a] * c - x[..., b] * s
        out[..., b] = x[..., b] * c + x[..., a] * s
    return out


def rotate_interleaved(x, positions, rot):
    return turn(x, positions, rot, [(2 * i, 2 * i + 1) for i in range(rot["dims"] // 2)])


def rotate_half(x, positions, rot):
    half = rot["dims"] // 2
    return turn(x, positions, rot, [(i, i + half) for i in range(half)])


# ------------------------------------------------------------------------------------------ latent attention
def latent_keys(h, w, spec, eps):
    """What a layer with its own cache keeps: normed latents (T, kv_rank) and the rotated key part (T, rot_dim)."""
    both = h @ w("dkv").T
    c, k = both[:, :spec["kv_rank"]], both[:, spec["kv_rank"]:]
    return rms_norm(c, w("dkv.norm"), eps), rotate_interleaved(k[:, None], torch.arange(len(h)), spec["rot"])[:, 0]


def latent_attention(h, w, spec, c, k_rot):
    """Mixer output for latents and rotated key parts that are this layer's own or another one's."""
    steps, heads, dim, rd, vdim = len(h), spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"]
    q = (h @ w("q").T).reshape(steps, heads, dim + rd)
    q_rot = rotate_interleaved(q[..., dim:], torch.arange(steps), spec["rot"])
    k, v = (c @ w("uk").T).reshape(steps, heads, dim), (c @ w("uv").T).reshape(steps, heads, vdim)
    hidden = torch.ones(steps, steps, dtype=torch.bool).triu(1)
    gate, out = torch.sigmoid(h @ w("g").T), []
    for n in range(heads):
        s = (q[:, n, :dim] @ k[:, n].T + q_rot[:, n] @ k_rot.T) * spec["scale"]
        out.append(torch.softmax(s.masked_fill(hidden, -math.inf), -1) @ v[:, n] * gate[:, n:n + 1])
    return torch.cat(out, 1) @ w("o").T


# ----------------------------------------------------------------------------------------- grouped attention
def visible(i, j, size, keep):
    return j <= i and (i - j < size or j < keep)


def sink_attention(q, k, v, scale, cap, size, keep, sink):
    """q (T, H, D), k (T, G, D), v (T, G, E): capped scores, a window beside the first tokens, and exp(sink) in the denominator."""
    steps, heads = q.shape[0], q.shape[1]
    rep = heads // k.shape[1]
    mask = torch.tensor([[visible(i, j, size, keep) for j in range(steps)] for i in range(steps)])
    out = torch.zeros(steps, heads, v.shape[-1], dtype=q.dtype)
    for h in range(heads):
        s = softcap(q[:, h] @ k[:, h // rep].T * scale, cap).masked_fill(~mask, -math.inf)
        s = torch.cat((s, sink[h].expand(steps, 1)), 1)
        out[:, h] = torch.softmax(s, -1)[:, :-1] @ v[:, h // rep]
    return out


def attention(h, w, spec, eps):
    steps, heads, kv, dim = len(h), spec["heads"], spec["kv_heads"], spec["dim"]
    proj = lambda name: h @ w(name).T + w(name + ".b")
    at = torch.arange(steps)
    q = rotate_half(rms_norm(proj("q"), w("q.norm"), eps).reshape(steps, heads, dim), at, spec["rot"])
    k = rotate_half(rms_norm(proj("k"), w("k.norm"), eps).reshape(steps, kv, dim), at, spec["rot"])
    v = proj("v").reshape(steps, kv, spec["vdim"])
    o = sink_attention(q, k, v, spec["scale"], spec["softcap"], spec["mask"]["size"], spec["mask"]["keep_first"], w("sink"))
    return o.reshape(steps, -1) @ w("o").T + w("o.b")


# ---------------------------------------------------------------------------------------------- feed-forward
def silu_glu(h, w_gate, w_up, w_down):
    g = h @ w_gate.T
    return (g * torch.sigmoid(g) * (h @ w_up.T)) @ w_down.T


def gelu(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def expert(h, w_up, w_down):
    return gelu(h @ w_up.T) @ w_down.T


def route(h, w_router, correction, top):
    """Chosen outputs (T, top) and their weights."""
    s = torch.softmax(h @ w_router.T, -1)
    chosen = torch.topk(s + correction, top, dim=-1).indices
    weight = s.gather(1, chosen)
    return chosen, weight / (weight.sum(-1, keepdim=True) + 1e-20)


def mixture(h, w, spec):
    """Routed experts, the last ``identity`` outputs of the router standing for the input itself, and a gated shared expert."""
    r = spec["router"]
    chosen, weight = route(h, w("router"), w("correction"), r["top"])
    out = torch.zeros_like(h)
    for t in range(len(h)):
        for e, a in zip(chosen[t].tolist(), weight[t]):
            out[t] += a * (h[t] if e >= r["experts"] else expert(h[t:t + 1], w(f"e{e}.up"), w(f"e{e}.down"))[0])
    return out + expert(h, w("shared.up"), w("shared.down")) * torch.sigmoid(h @ w("shared.sg").T)


class Oracle:
    def __init__(self, config, tensors, dtype=torch.float64):
        self.cfg, self.dtype = config, dtype
        self.t = {k: v.to(dtype) for k, v in tensors.items()}

    def residuals(self, tokens):
        """The residual stream after every layer: [layers, tokens, width]."""
        cfg, t = self.cfg, self.t
        eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
        x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
        out, kept = [], {}
        for i, layer in enumerate(cfg["layers"]):
            pre, spec, mlp = f"l{i}.", layer["mixer"], layer.get("mlp")
            w = lambda name: t[pre + "mix." + name]
            h = centred_norm(x, t[pre + "norm1"], eps)
            if layer["type"] == "attention":
                x = x + m * attention(h, w, spec, eps)
            else:
                src = spec.get("kv_from")
                if src is None:
                    src, kept[i] = i, latent_keys(h, w, spec, eps)
                x = x + m * latent_attention(h, w, spec, *kept[src])
            if mlp:
                h, w = centred_norm(x, t[pre + "norm2"], eps), (lambda name: t[pre + "mlp." + name])
                x = x + m * (silu_glu(h, w("gate"), w("up"), w("down")) if mlp["kind"] == "dense" else mixture(h, w, mlp))
            out.append(x)
        return torch.stack(out)

    def logits(self, tokens):
        x = self.residuals(tokens)[-1]
        return softcap(centred_norm(x, self.t["final.norm"], self.cfg["norm"]["eps"]) @ self.t["head"].T, self.cfg["logit_softcap"])
