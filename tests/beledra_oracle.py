"""Plain, slow statement of the Beledra design: one function per mechanism, loops where loops are clearest.

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


# ------------------------------------------------------------------------------------- matrix memory (mLSTM)
def log_gates(h, w_i, b_i, w_f, b_f, cap):
    """Logarithms of the input and forget gates, (T, heads) each: the pre-activations are capped softly at +-cap."""
    soft = lambda z: cap * torch.tanh(z / cap)
    return soft(h @ w_i.T + b_i), torch.nn.functional.logsigmoid(soft(h @ w_f.T + b_f))


def mlstm_scan(q, k, v, i, f):
    """q, k (T, H, D), v (T, H, E), log gates i, f (T, H): one token at a time, with the running maximum m that keeps the
    exponentials in range (it starts at zero)."""
    steps, heads, dim = q.shape
    out = torch.zeros(steps, heads, v.shape[-1], dtype=q.dtype)
    S = torch.zeros(heads, dim, v.shape[-1], dtype=q.dtype)
    n = torch.zeros(heads, dim, dtype=q.dtype)
    m = torch.zeros(heads, dtype=q.dtype)
    for t in range(steps):
        new = torch.maximum(f[t] + m, i[t])
        keep, take = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        m = new
        S = keep[:, None, None] * S + take[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + take[:, None] * k[t]
        low = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out[t] = torch.einsum("hde,hd->he", S, q[t]) / low[:, None]
    return out


def mlstm(h, w, spec, eps):
    """The whole mixer for one sequence h (T, width); ``w(name)`` gives a weight."""
    steps, heads, dim, vdim = h.shape[0], spec["heads"], spec["dim"], spec["vdim"]
    q = (h @ w("q").T).reshape(steps, heads, dim) * dim ** -0.5
    k = (h @ w("k").T).reshape(steps, heads, dim)
    v = (h @ w("v").T).reshape(steps, heads, vdim)
    i, f = log_gates(h, w("i"), w("i.b"), w("f"), w("f.b"), spec["gate_cap"])
    o = rms(mlstm_scan(q, k, v, i, f), eps).reshape(steps, heads * vdim) * w("norm")
    return (o * torch.sigmoid(h @ w("g").T)) @ w("o").T


# ------------------------------------------------------------------------------------------------- attention
def distance_bucket(n, rows, far):
    """Row of the distance table for a key ``n`` tokens back: exact for near keys, logarithmic up to ``far``."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_bias(table, far, steps):
    """(H, T, T): table[bucket(i - j), h] for j <= i (zero elsewhere)."""
    out = torch.zeros(table.shape[1], steps, steps, dtype=table.dtype)
    for i in range(steps):
        for j in range(i + 1):
            out[:, i, j] = table[distance_bucket(i - j, table.shape[0], far)]
    return out


def window_attention(q, k, v, scale, size, bias=None):
    """Softmax attention: q (T, H, D), k (T, G, D), v (T, G, E); query head h reads head h // (H / G); position i sees j with
    0 <= i - j < size; ``bias`` (H, T, T) is added to the scaled scores."""
    steps, heads = q.shape[0], q.shape[1]
    rep = heads // k.shape[1]
    i = torch.arange(steps)
    seen = (i[:, None] - i[None, :] >= 0) & (i[:, None] - i[None, :] < size)
    out = torch.zeros(steps, heads, v.shape[-1], dtype=q.dtype)
    for h in range(heads):
        s = q[:, h] @ k[:, h // rep].T * scale
        if bias is not None:
            s = s + bias[h]
        out[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, h // rep]
    return out


def attention(h, w, spec, eps):
    steps, heads, kv, dim, vdim = h.shape[0], spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
    q = rms_norm((h @ w("q").T).reshape(steps, heads, dim), w("q.norm"), eps)
    k = rms_norm((h @ w("k").T).reshape(steps, kv, dim), w("k.norm"), eps)
    v = (h @ w("v").T).reshape(steps, kv, vdim)
    o = window_attention(q, k, v, spec["scale"], spec["mask"]["size"], distance_bias(w("rel"), spec["bias_max"], steps))
    return o.reshape(steps, heads * vdim) @ w("o").T


def yarn(rot):
    """Frequencies of the rotated pairs and the factor on cos and sin."""
    dims, base, sc = rot["dims"], float(rot["base"]), rot.get("scaling")
    freq = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if not sc:
        return freq, 1.0
    dim_of = lambda turns: dims * math.log(sc["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(dim_of(sc["fast"])), 0), min(math.ceil(dim_of(sc["slow"])), dims - 1)
    out = []
    for i, f in enumerate(freq):
        ramp = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / sc["factor"] * ramp + f * (1 - ramp))
    return out, 0.1 * math.log(sc["factor"]) + 1.0


def rotate_half(x, positions, freq, gain, dims):
    """Rotary embedding of (T, heads, dim): dimension i < dims/2 is paired with i + dims/2, the rest stays."""
    half, out = dims // 2, x.clone()
    for i in range(half):
        angle = positions.double() * freq[i]
        c, s = (gain * torch.cos(angle)).to(x.dtype)[:, None], (gain * torch.sin(angle)).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


def normed_rotated(x, weight, rot, eps):
    """x (T, heads * maps, dim): norm per head and map, then rotation."""
    freq, gain = yarn(rot)
    return rotate_half(rms_norm(x, weight, eps), torch.arange(x.shape[0]), freq, gain, rot["dims"])


def differential(a1, a2, lq1, lk1, lq2, lk2, diff, eps):
    """Difference of the two maps' outputs (T, H, E), normed per head."""
    lam = torch.exp((lq1 * lk1).sum()) - torch.exp((lq2 * lk2).sum()) + diff
    return rms(a1 - lam * a2, eps) * (1 - diff)


def keys_values(h, w, spec, eps):
    steps, kv = h.shape[0], spec["kv_heads"]
    k = normed_rotated((h @ w("k").T).reshape(steps, kv * 2, spec["dim"]), w("k.norm"), spec["rot"], eps)
    return k, (h @ w("v").T).reshape(steps, kv, spec["vdim"])


def attention_2(h, w, spec, eps, k, v):
    """Differential attention with keys k (T, kv * 2, dim) and values v (T, kv, vdim), its own or another layer's."""
    steps, heads = h.shape[0], spec["heads"]
    q = normed_rotated((h @ w("q").T).reshape(steps, heads * 2, spec["dim"]), w("q.norm"), spec["rot"], eps)
    a = [window_attention(q[:, m::2], k[:, m::2], v, spec["scale"], spec["mask"]["size"]) for m in (0, 1)]
    o = differential(*a, w("lq1"), w("lk1"), w("lq2"), w("lk2"), spec["diff"], eps)
    return (o.reshape(steps, heads * spec["vdim"]) * torch.sigmoid(h @ w("g").T)) @ w("o").T


# ----------------------------------------------------------------------------------------------- feed-forward
def relu_glu(x, w_gate, w_up, w_down):
    return (torch.relu(x @ w_gate.T) * (x @ w_up.T)) @ w_down.T


class Oracle:
    def __init__(self, config, tensors, dtype=torch.float64):
        self.cfg, self.dtype = config, dtype
        self.t = {k: v.to(dtype) for k, v in tensors.items()}

    def residuals(self, tokens):
        """The residual stream after every layer: [layers, tokens, width]."""
        cfg, t = self.cfg, self.t
        eps = cfg["norm"]["eps"]
        x = t["embed"][torch.as_tensor(tokens, dtype=torch.long)]
        out, kept = [], {}
        for i, layer in enumerate(cfg["layers"]):
            pre, spec = f"l{i}.", layer["mixer"]
            w = lambda name: t[pre + "mix." + name]
            if layer["type"] == "mlstm":
                y = mlstm(x, w, spec, eps)
            elif layer["type"] == "attention":
                y = attention(x, w, spec, eps)
            else:
                if spec.get("kv_from") is None:
                    kept[i] = keys_values(x, w, spec, eps)
                    k, v = kept[i]
                else:
                    k, v = kept[spec["kv_from"]]
                y = attention_2(x, w, spec, eps, k, v)
            x = x + rms_norm(y, t[pre + "norm1"], eps)
            if layer.get("mlp"):
                y = relu_glu(x, *(t[pre + "mlp." + k] for k in ("gate", "up", "down")))
                x = x + rms_norm(y, t[pre + "norm2"], eps)
            out.append(x)
        return torch.stack(out)

    def logits(self, tokens):
        x = self.residuals(tokens)[-1]
        return rms_norm(x, self.t["final.norm"], self.cfg["norm"]["eps"]) @ self.t["head"].T
