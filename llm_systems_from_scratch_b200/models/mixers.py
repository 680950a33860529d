"""Sublayers of layered decoders: token mixers and feed-forwards that a model puts together by configuration.

Each class takes its sizes and constants as arguments, packs its weights for the kernels (matrices that read the same
input become one product; heads are padded to what the kernels tile by) and runs one step of the engine:

* a mixer is called with its input rows ``h``, the fp32 residual stream ``x``, the ``StepBatch`` and its own part of the
  cache (``cache_spec()`` says what that is).  It adds its output to ``x`` in the epilogue of its output projection, or
  returns it when ``x`` is None (designs that norm a sublayer's output before they add it)
* a feed-forward does the same, or returns outputs that the next pass over the residual stream adds (``ops.mixer_ops``:
  ``residual_norm``, ``add_normed``)

What a sublayer adds to ``x`` it multiplies with its ``gain``.  Designs that gate a sublayer's output before they norm it give the gate's
weights to the sublayer (``out_gate``), where their product joins those of the same input; it then returns (output, gate).

``get(name)`` gives a weight in its stored layout ([out, in])."""
from __future__ import annotations

import math

import torch

from ..ops import mixer_ops as mo
from ..serving.kv_cache import PagedSpec, Parts, SharedSpec, StateSpec


def _head_pad(w, heads: int, rows: int, to: int):
    """[heads * rows, in] -> [heads * to, in] with zero rows after each head's."""
    if rows == to:
        return w
    out = torch.zeros((heads, to, w.shape[1]), dtype=w.dtype, device=w.device)
    out[:, :rows] = w.view(heads, rows, -1)
    return out.view(heads * to, -1)


def _expect(name: str, t, *shape):
    if tuple(t.shape) != shape:
        raise ValueError(f"{name} has shape {tuple(t.shape)}, expected {shape}")
    return t


def _project(y, w_o, x, gain: float = 1.0, bias=None):
    """The output projection, into the residual stream or returned."""
    return mo.linear(y, w_o, bias=bias) if x is None else mo.linear(y, w_o, out=x, accumulate=True, alpha=gain, bias=bias)


def _align(n: int, to: int) -> int:
    return -(-n // to) * to


def _row_pad(w, to: int):
    """Zero rows up to ``to``."""
    return w if w.shape[0] == to else torch.cat((w, torch.zeros((to - w.shape[0], w.shape[1]), dtype=w.dtype, device=w.device)))


class InputProducts:
    """Weights that read a sublayer's input, as one matrix: each part starts at a multiple of 8 columns (``at``), biases where there are any."""

    def __init__(self, parts: dict, biases: dict, dtype, device):
        rows, self.at, n = [], {}, 0
        bias = torch.zeros(sum(_align(len(w), 8) for w in parts.values()), dtype=torch.float32)
        for name, w in parts.items():
            self.at[name] = slice(n, n + len(w))
            if biases.get(name) is not None:
                bias[n:n + len(w)] = biases[name].float()
            rows.append(_row_pad(w, _align(len(w), 8)))
            n += len(rows[-1])
        self.w = mo.padded_weight(torch.cat(rows), dtype, device)
        self.bias = bias.to(device) if any(b is not None for b in biases.values()) else None

    def __call__(self, h):
        return mo.linear(h, self.w, bias=self.bias)


def conv_filter(get, names, sizes, taps: int, dtype, device):
    """The filters of some projections, (channels, taps) each, as one matrix (taps, channels)."""
    if taps < 1:
        raise ValueError("a convolution has one tap at least")
    both = torch.cat([_expect(n + ".conv", get(n + ".conv"), size, taps) for n, size in zip(names, sizes)])
    return both.t().to(device=device, dtype=dtype).contiguous()


class LatentAttention:
    """Attention whose keys and values are linear images of one cached latent per token.

    q = W_uq rms_norm(W_dq h), or W_q h without a ``q_rank``; c = rms_norm(W_dkv h), k_h = W_uk,h c, v_h = W_uv,h c,
    softmax(scale q.k) over the last ``window`` positions (0 = all), heads multiplied by sigmoid(W_g h) (``gate``: "elements", or
    one number per head: "heads"), then W_o.  The cache holds c.  Optional parts:

    * ``rot_dim`` / ``rope``: every head's query has rot_dim more rows, which are rotated (interleaved pairs); W_dkv has rot_dim more
      rows, a rotated key part shared by all heads, cached behind c
    * ``kv_from``: latents and key parts of that earlier layer run instead of its own"""

    def __init__(self, get, width: int, heads: int, dim: int, vdim: int, q_rank: int | None, kv_rank: int, scale: float, window: int,
                 eps: float, dtype, device, rot_dim: int = 0, rope=None, kv_from: int | None = None, gate: str = "elements",
                 gain: float = 1.0):
        if rot_dim % 2 or (rot_dim and rope is None):
            raise ValueError("the rotated dimensions come in pairs and need angles")
        if gate not in ("elements", "heads"):
            raise ValueError(f"unknown gate {gate!r}")
        self.heads, self.dim, self.vdim, self.q_rank, self.kv_rank = heads, dim, vdim, q_rank, kv_rank
        self.rot, self.rope, self.kv_from, self.gain = int(rot_dim), rope, kv_from, float(gain)
        self.scale, self.window, self.eps = float(scale), int(window), float(eps)
        self.latent, self.rp = mo.pitch(kv_rank), mo.pitch(rot_dim)             # cached parts, zero padded
        self.cached = self.latent + self.rp
        w = lambda name, *shape: _expect(name, get(name), *shape)
        pack = lambda t: mo.padded_weight(t, dtype, device)
        # the tensor-core prefill takes heads up to 128 whose columns are multiplied 16 at a time; elsewhere a head only has to start on
        # a 16-byte boundary
        self.tiles = (dtype == torch.bfloat16 and torch.device(device).type == "cuda" and max(dim, vdim) <= 128 and rot_dim <= 64
                      and scale > 0)
        self.qp, self.vp = _align(dim, 16) if self.tiles else mo.pitch(dim), mo.pitch(vdim)
        # queries: the unrotated parts of all heads, then the rotated ones
        own = w("uq", heads * (dim + rot_dim), q_rank) if q_rank is not None else w("q", heads * (dim + rot_dim), width)
        own = own.view(heads, dim + rot_dim, -1)
        q = _head_pad(own[:, :dim].reshape(heads * dim, -1), heads, dim, self.qp)
        if rot_dim:
            q = torch.cat((q, _head_pad(own[:, dim:].reshape(heads * rot_dim, -1), heads, rot_dim, self.rp)))
        parts, at = [], 0
        self.w_uq = self.n_q = None
        if q_rank is not None:
            parts.append(w("dq", q_rank, width))
            self.w_uq, self.n_q = pack(q), w("dq.norm", q_rank).to(device=device, dtype=dtype).contiguous()
        else:
            parts.append(q)
        self.kv_col = self.k_col = self.n_kv = None
        if kv_from is None:
            dkv = w("dkv", kv_rank + rot_dim, width)
            self.kv_col = sum(len(p) for p in parts)
            parts.append(dkv[:kv_rank])
            if rot_dim:
                parts[-1] = _row_pad(parts[-1], self.latent)
                self.k_col = self.kv_col + self.latent
                parts.append(_row_pad(dkv[kv_rank:], self.rp))
            self.n_kv = w("dkv.norm", kv_rank).to(device=device, dtype=dtype).contiguous()
        self.gate_col = sum(len(p) for p in parts)
        parts.append(w("g", heads * vdim if gate == "elements" else heads, width))
        self.w_in = pack(torch.cat(parts))
        uk, uv = w("uk", heads * dim, kv_rank), w("uv", heads * vdim, kv_rank)
        ukt = torch.zeros((heads, self.latent, self.qp), dtype=uk.dtype, device=uk.device)        # q_h -> latent space: W_uk,h^T
        ukt[:, :kv_rank, :dim] = uk.view(heads, dim, kv_rank).transpose(1, 2)
        self.w_ukt = pack(ukt.reshape(heads * self.latent, self.qp))
        uvp = torch.zeros((heads * vdim, self.latent), dtype=uv.dtype, device=uv.device)
        uvp[:, :kv_rank] = uv
        self.w_uv = pack(uvp)
        if self.tiles:
            kv = torch.zeros((heads * (self.qp + self.vp), self.latent), dtype=uk.dtype, device=uk.device)
            kv[:heads * self.qp, :kv_rank] = _head_pad(uk, heads, dim, self.qp)
            kv[heads * self.qp:, :kv_rank] = _head_pad(uv, heads, vdim, self.vp)
            self.w_ukv = pack(kv)
        self.w_o = pack(w("o", width, heads * vdim))

    def cache_spec(self):
        return PagedSpec(self.cached) if self.kv_from is None else SharedSpec(self.kv_from)

    def __call__(self, h, x, batch, cache):
        heads, n, rows = self.heads, batch.n_single, batch.n_rows
        proj = mo.linear(h, self.w_in)
        q = proj
        if self.q_rank is not None:
            cq = mo.latent_norm_append(proj, self.n_q, self.n_kv, self.eps, cache, batch.slots)
            q = mo.linear(cq, self.w_uq)
        gate = proj[:, self.gate_col:]
        o = mo.rows_buffer(rows, heads * self.vdim, h.dtype, h.device)
        absorbed = n if self.tiles else rows             # rows whose queries move into latent space
        ql = None
        if absorbed:
            ql = torch.empty((absorbed, heads * self.cached), dtype=h.dtype, device=h.device)
            mo.gemm_heads(q[:absorbed], self.w_ukt, heads, self.qp, self.latent, out=ql, c_step=self.cached)
        if self.rot:
            mo.latent_rotate(q, heads * self.qp, self.rp, proj, self.kv_col if self.q_rank is None else None, self.k_col, self.n_kv, ql,
                             cache, self.rope.table, batch.positions, batch.slots, heads, self.kv_rank, self.latent, self.rot, self.eps)
        if n:
            ol = mo.latent_decode(ql[:n], cache, batch.positions[:n], batch.slots[:n], batch.tables[:n], heads, self.window, self.scale,
                                  vwidth=self.latent)
            mo.gemm_heads(ol, self.w_uv, heads, self.latent, self.vdim, out=o[:n], gate=gate[:n])
        if rows > n and self.tiles:
            self._portions(q[n:], gate[n:], o[n:], batch, cache)
        elif rows > n:
            ol = mo.latent_attention_rows(ql[n:], cache, batch.row_seq[n:], batch.positions[n:], batch.slots[n:], batch.tables, heads,
                                          self.window, self.scale, self.latent)
            mo.gemm_heads(ol, self.w_uv, heads, self.latent, self.vdim, out=o[n:], gate=gate[n:])
        return _project(o, self.w_o, x, self.gain)

    def _portions(self, q, gate, o, batch, cache):
        """Keys and values of everything the portions can see, expanded from the cached latents."""
        heads = self.heads
        cu_k, first, total, _ = batch.key_ranges(self.window)
        key = (cache.data_ptr(), self.window)            # layers that share a cache share its packed rows
        if key not in batch.gathered:
            batch.gathered[key] = mo.latent_gather(cache, cu_k, first, batch.tables[batch.n_single:], total)
        c = batch.gathered[key]
        kv = mo.linear(c[:, :self.latent], self.w_ukv)
        rot = (c, self.rot, heads * self.qp, self.rp, self.latent) if self.rot else None
        mo.window_attention(q, kv, batch.cu, cu_k, batch.max_portion, heads, self.dim, self.vdim, self.window, self.scale, o, gate,
                            (self.qp, self.qp, self.vp, heads * self.qp), rot)


class Retention:
    """Attention without softmax whose memory is a decaying matrix per head: S <- d S + k v^T, read by q.  q and k are
    rotated (rotate-half over the first ``rot_dims`` dimensions); heads are divided by their root mean square, multiplied
    by silu(W_g h), then W_o.  The state is fp32."""

    MIN_CHUNKED = 8            # the longest portion of a step from which the chunked kernel is used

    def __init__(self, get, width: int, heads: int, dim: int, vdim: int, decay, rot_dims: int, eps: float, rope, dtype, device):
        self.heads, self.dim, self.vdim, self.rot, self.eps = heads, dim, vdim, int(rot_dims), float(eps)
        if len(decay) != heads:
            raise ValueError(f"{len(decay)} decays for {heads} heads")
        if self.rot % 2 or self.rot > dim:
            raise ValueError("the rotated dimensions must be even in number and fit the head")
        w = lambda name, *shape: _expect(name, get(name), *shape)
        self.w_in = mo.padded_weight(torch.cat((w("q", heads * dim, width), w("k", heads * dim, width),
                                                w("v", heads * vdim, width), w("g", heads * vdim, width))), dtype, device)
        self.w_o = mo.padded_weight(w("o", width, heads * vdim), dtype, device)
        self.decay = torch.tensor([float(d) for d in decay], dtype=torch.float32, device=device)
        self.powers = None                     # for prompts on the tensor cores, where sizes and decays allow it
        if torch.device(device).type == "cuda" and mo.chunkable(dtype, dim, vdim, self.rot):
            self.powers = mo.retention_powers(decay, device)
        self.rope = rope                       # RotaryTable of the model's base and dims, None without rotation

    def cache_spec(self):
        return StateSpec((self.heads, self.dim, self.vdim))

    def __call__(self, h, x, batch, state):
        n = batch.n_single
        proj = mo.linear(h, self.w_in)
        y = mo.rows_buffer(h.shape[0], self.heads * self.vdim, h.dtype, h.device)
        table = self.rope.table if self.rope is not None else None
        run = lambda rows, slots, cu, spans: mo.retention(
            proj[rows], state, slots, cu, spans, batch.positions[rows], table, self.decay, self.heads, self.dim, self.vdim,
            self.rot, self.eps, y[rows])
        if n:
            run(slice(0, n), batch.state_slots[:n], None, [(i, i + 1) for i in range(n)] if not h.is_cuda else None)
        if batch.n_rows > n and self.powers is not None and batch.max_portion >= self.MIN_CHUNKED:
            mo.retention_chunked(proj[n:], state, batch.state_slots[n:], batch.cu, batch.positions[n:], table, self.powers,
                                 self.heads, self.dim, self.vdim, self.rot, self.eps, y[n:])
        elif batch.n_rows > n:
            run(slice(n, batch.n_rows), batch.state_slots[n:], batch.cu, batch.spans)
        return _project(y, self.w_o, x)


class MatrixMemory:
    """Matrix memory with exponential gates (mLSTM of xLSTM): per head S <- f S + i k v^T and a normaliser n <- f n + i k, kept
    in range by a running maximum m of the log gates that starts at zero; o = S^T q / (max(|n . q|, exp(-m)) + 1e-6).

    The log gates are capped softly (cap tanh(z / cap)); heads are divided by their root mean square, multiplied by the
    weight ``norm`` and by sigmoid(W_g h), then W_o.  S, n and m are fp32 and share one state slot per request."""

    MIN_CHUNKED = 8            # the longest portion of a step from which the chunked kernel is used

    def __init__(self, get, width: int, heads: int, dim: int, vdim: int, gate_cap: float, eps: float, dtype, device):
        self.heads, self.dim, self.vdim, self.cap, self.eps = heads, dim, vdim, float(gate_cap), float(eps)
        w = lambda name, *shape: _expect(name, get(name), *shape)
        pack = lambda *ts: mo.padded_weight(torch.cat(ts), dtype, device)
        self.w_in = pack(w("q", heads * dim, width), w("k", heads * dim, width), w("v", heads * vdim, width),
                         w("g", heads * vdim, width))
        self.w_gates = pack(w("i", heads, width), w("f", heads, width))
        self.b_gates = torch.cat((w("i.b", heads), w("f.b", heads))).to(device=device, dtype=torch.float32).contiguous()
        self.norm = w("norm", heads * vdim).to(device=device, dtype=dtype).contiguous()
        self.w_o = mo.padded_weight(w("o", width, heads * vdim), dtype, device)
        self.chunked = torch.device(device).type == "cuda" and mo.mlstm_chunkable(dtype, dim, vdim)
        self.one_pass = mo.mlstm_steps(dim, vdim)          # a decode step takes the gates' products itself

    def cache_spec(self):
        return StateSpec((self.heads, mo.mlstm_state(self.dim, self.vdim)))

    def __call__(self, h, x, batch, state):
        n = batch.n_single
        proj = mo.linear(h, self.w_in)
        y = mo.rows_buffer(h.shape[0], self.heads * self.vdim, h.dtype, h.device)

        def run(rows, seqs, cu, spans, chunked):
            # the recurrence takes the gates in 32-bit
            gates = (h[rows], self.w_gates) if cu is None and self.one_pass else mo.linear(h[rows], self.w_gates, out_dtype=torch.float32)
            mo.mlstm(proj[rows], gates, self.b_gates, self.norm, state, batch.state_slots[seqs], cu, spans,
                     batch.positions[rows], self.heads, self.dim, self.vdim, self.cap, self.eps, y[rows], chunked)
        if n:
            run(slice(0, n), slice(0, n), None, [(i, i + 1) for i in range(n)] if not h.is_cuda else None, False)
        if batch.n_rows > n:
            run(slice(n, batch.n_rows), slice(n, None), batch.cu, batch.spans, self.chunked and batch.max_portion >= self.MIN_CHUNKED)
        return _project(y, self.w_o, x)


class GroupedAttention:
    """Softmax attention of grouped heads under a sliding window: query head h reads key/value head h // (heads / kv_heads).

    Queries and keys are RMS-normed (weights ``q.norm`` / ``k.norm``; ``norm`` "head": per head, "projection": over all heads at
    once), rotated in their first ``rot_dims`` dimensions (``rope``), scored with ``scale``.  Optional parts:

    * ``keep``: the first ``keep`` positions of a sequence stay visible whatever the window
    * ``softcap``: scores are capped softly, cap tanh(score / cap)
    * ``sink``: exp(sink_h), a number per head, joins the softmax's denominator
    * ``biased``: q, k, v and o have biases (``q.b`` ...)
    * ``bias_max``: a table ``rel`` (buckets, heads) adds a bias per distance to the scaled scores, exact for near keys and
      logarithmic up to ``bias_max``
    * ``difference`` (with ``out_scale``): two maps per head over the same values (queries and keys have twice the rows, laid
      out head by head); the output is first map - difference * second map, RMS-normed per head, times ``out_scale``
    * ``gated``: heads are multiplied by sigmoid(W_g h), element by element, or with one number per head (``gated`` "heads")
    * ``chunked``: a query sees the keys of its own chunk of ``window`` positions instead
    * ``slopes``: slope_h * distance comes off the scaled scores
    * ``conv`` (with ``norm`` None, no rotation): projections pass a short convolution of that many taps; then
      * ``temp``: scores are multiplied by a number per head
      * ``mix_from`` (an earlier layer run, or None): values are mixed with that run's of the same token by the weight ``vmix``
    * ``kv_from``: keys and values of that earlier layer run instead of its own

    The cache holds the normed, rotated keys and the values of a token as one vector, every head padded to 8 elements."""

    def __init__(self, get, width: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, window: int, eps: float,
                 dtype, device, bias_max: float | None = None, rope=None, rot_dims: int = 0, difference: float | None = None,
                 out_scale: float = 1.0, gated: bool = False, kv_from: int | None = None, keep: int = 0, softcap: float | None = None,
                 sink: bool = False, biased: bool | str = False, norm: str | None = "head", gain: float = 1.0, chunked: bool = False,
                 slopes=None, conv: int = 0, temp: bool = False, mix_from: int | None = None, out_gate=None):
        self.gated, self.kv_from, self.rope, self.gain = bool(gated), kv_from, rope, float(gain)
        self.taps, self.mix_from, self.mix, self.gates_output = int(conv), mix_from, 0.0, out_gate is not None
        if heads % kv_heads:
            raise ValueError("the query heads must share the key heads evenly")
        if rot_dims % 2 or rot_dims > dim:
            raise ValueError("the rotated dimensions must be even in number and fit the head")
        if norm not in ("head", "projection", None):
            raise ValueError(f"unknown norm {norm!r}")
        maps = 1 if difference is None else 2
        if maps == 2 and (sink or norm == "projection" or slopes is not None):
            raise ValueError("sinks, slopes and norms over a projection are those of a single map")
        if bool(conv) != (norm is None) or (conv and (maps == 2 or rot_dims or kv_from is not None)):
            raise ValueError("projections are normed, or pass a convolution and are neither rotated nor shared")
        if (temp or mix_from is not None) and not conv:
            raise ValueError("factors of the scores and mixed values come with the convolution")
        if (chunked and keep) or (slopes is not None and (softcap or bias_max is not None)):
            raise ValueError("chunks keep no first tokens, and slopes go with neither caps nor tables")
        w = lambda name, *shape: _expect(name, get(name), *shape)
        rows = {"q": heads * maps * dim}
        if kv_from is None:
            rows.update({"k": kv_heads * maps * dim, "v": kv_heads * vdim})
        qkv = torch.cat([w(name, n, width) for name, n in rows.items()])
        parts, biases = {"qkv": qkv}, {}
        if gated:
            parts["g"] = w("g", heads if gated == "heads" else heads * vdim, width)
        if out_gate is not None:
            parts["out"], biases["out"] = out_gate
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.b_o = None
        if biased:                                       # "inputs": q, k and v alone
            biases["qkv"] = torch.cat([w(name + ".b", n) for name, n in rows.items()])
            self.b_o = f32(w("o.b", width)) if biased != "inputs" else None
        self.inputs = InputProducts(parts, biases, dtype, device)
        self.w_o = mo.padded_weight(w("o", width, heads * vdim), dtype, device)
        if norm is not None:
            vec = lambda name, n: w(name, dim if norm == "head" else n * dim).to(device=device, dtype=dtype).contiguous()
            self.n_q, self.n_k = vec("q.norm", heads), vec("k.norm", kv_heads) if kv_from is None else None
        if conv:
            self.channels = len(qkv)
            self.filter = conv_filter(get, rows, rows.values(), self.taps, dtype, device)
            self.temp = f32(w("temp", heads)) if temp else torch.ones(heads, dtype=torch.float32, device=device)
            if mix_from is not None:
                self.mix = float(w("vmix"))
        bias = None
        if bias_max is not None:
            rel = get("rel")
            if rel.shape[1] != heads:
                raise ValueError(f"rel has shape {tuple(rel.shape)}, expected {heads} columns")
            bias = distance_table(rel, bias_max, window).to(device)
        self.shape = mo.AttentionShape(heads, kv_heads, maps, dim, vdim, rot_dims, float(scale), int(window), float(eps),
                                       float(difference or 0.0), float(out_scale), bias, int(keep), float(softcap or 0.0),
                                       f32(w("sink", heads)) if sink else None, norm == "projection",
                                       None if slopes is None else torch.tensor(slopes, dtype=torch.float32, device=device), bool(chunked),
                                       gated == "heads")
        self.tensor_cores = torch.device(device).type == "cuda" and mo.attention_tiles(self.shape, dtype)

    def cache_spec(self):
        own = PagedSpec(self.shape.cache_width)
        if self.taps:
            ring = StateSpec((self.taps, self.channels), "activations")
            return Parts((own, ring) if self.mix_from is None else (own, ring, SharedSpec(self.mix_from)))
        return own if self.kv_from is None else SharedSpec(self.kv_from)

    def _convolved(self, u, batch, cache):
        """Queries behind the convolution; keys and values are in the cache then.  -> queries, the paged pool"""
        pool, ring, *first = cache
        parts = mo.step_parts(batch)
        q = [mo.conv_attend(u[rows], self.filter, ring, at, self.shape, self.temp, pool, first[0][0] if first else None, self.mix)
             for rows, at in parts]
        return q[0] if len(q) == 1 else torch.cat(q), pool

    def __call__(self, h, x, batch, cache):
        s, n = self.shape, batch.n_single
        proj = self.inputs(h)
        at = self.inputs.at
        if self.taps:
            q, cache = self._convolved(proj[:, at["qkv"]], batch, cache)
        else:
            q = mo.attention_prepare(proj, s, self.n_q, self.n_k, self.rope.table if self.rope is not None else None,
                                     batch.positions, batch.slots, cache)
        o = mo.rows_buffer(h.shape[0], s.heads * s.vdim, h.dtype, h.device)
        gate = proj[:, at["g"]] if self.gated else None
        part = lambda rows: None if gate is None else gate[rows]
        if n:
            one = slice(0, n)
            mo.attention_decode(q[one], s, cache, batch.positions[one], batch.slots[one], batch.tables[one], o[one], part(one))
        if batch.n_rows > n:
            rest = slice(n, batch.n_rows)
            if self.tensor_cores and mo.attention_pages(cache.shape[1]):
                mo.attention_portions(q[rest], s, cache, batch.positions[rest], batch.cu, batch.max_portion, batch.tables[n:],
                                      o[rest], part(rest))
            else:
                mo.attention_rows(q[rest], s, cache, batch.row_seq[rest], batch.positions[rest], batch.slots[rest],
                                  batch.tables, o[rest], part(rest))
        y = _project(o, self.w_o, x, self.gain, self.b_o)
        return (y, proj[:, at["out"]]) if self.gates_output else y


class DeltaRule:
    """Gated delta rule: per head S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q, with unit q (times dim^(-1/2)) and k shared by
    heads / kv_heads heads, a decay g = exp(-exp(A_log) softplus(W_a h + dt_bias)) and beta = sigmoid(W_b h) per head.

    Projections of q, k and v pass a short convolution of ``taps`` taps and silu; heads are divided by their root mean square, multiplied
    by the weight ``norm`` and by silu(W_g h), then W_o.  S is fp32; a request's state slot holds it and the convolution's last inputs."""

    MIN_CHUNKED = 8            # the longest portion of a step from which the chunked kernels are used

    def __init__(self, get, width: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, eps: float, dtype, device, out_gate=None):
        if heads % kv_heads:
            raise ValueError("the heads must share the keys evenly")
        self.heads, self.kv_heads, self.dim, self.vdim, self.eps = heads, kv_heads, dim, vdim, float(eps)
        w = lambda name, *shape: _expect(name, get(name), *shape)
        rows = {"q": kv_heads * dim, "k": kv_heads * dim, "v": heads * vdim}
        parts = {"qkv": torch.cat([w(name, n, width) for name, n in rows.items()]), "g": w("g", heads * vdim, width)}
        self.channels, self.gates_output, biases = len(parts["qkv"]), out_gate is not None, {}
        if out_gate is not None:
            parts["out"], biases["out"] = out_gate
        self.inputs = InputProducts(parts, biases, dtype, device)
        self.w_ab = mo.padded_weight(torch.cat((w("a", heads, width), w("b", heads, width))), dtype, device)
        f32 = lambda t: t.to(device=device, dtype=torch.float32).contiguous()
        self.decay, self.dt = f32(-torch.exp(w("A_log", heads).double())), f32(w("dt_bias", heads))
        self.norm = w("norm", vdim).to(device=device, dtype=dtype).contiguous()
        self.filter = conv_filter(get, rows, rows.values(), taps, dtype, device)
        self.w_o = mo.padded_weight(w("o", width, heads * vdim), dtype, device)
        self.one_pass = mo.delta_steps(dim, vdim)          # a decode step takes the gates' products and the convolution itself
        self.chunked = torch.device(device).type == "cuda" and mo.delta_chunkable(dtype, dim, vdim)

    def cache_spec(self):
        return Parts((StateSpec((self.heads, self.dim, self.vdim)), StateSpec((len(self.filter), self.channels), "activations")))

    def __call__(self, h, x, batch, cache):
        state, ring = cache
        proj = self.inputs(h)
        at = self.inputs.at
        u, gate = proj[:, at["qkv"]], proj[:, at["g"]]
        y = mo.rows_buffer(h.shape[0], self.heads * self.vdim, h.dtype, h.device)
        for rows, part in mo.step_parts(batch):
            run = lambda c, ab, **kw: mo.delta_rule(c, gate[rows], ab, self.decay, self.dt, self.norm, state, part, self.kv_heads, self.eps, y[rows], **kw)
            if part.cu is None and self.one_pass:
                run(u[rows], (h[rows], self.w_ab), conv=(self.filter, ring))
                continue
            ab = mo.linear(h[rows], self.w_ab, out_dtype=torch.float32)        # the recurrence takes the gates in 32-bit
            c = mo.short_conv(u[rows], self.filter, ring, part, mo.rows_buffer(len(part.positions), self.channels, h.dtype, h.device), silu=True)
            chunks = part.cu is not None and self.chunked and batch.max_portion >= self.MIN_CHUNKED
            run(c, ab, chunks=batch.chunk_ranges(mo.DELTA_CHUNK) if chunks else None)
        out = _project(y, self.w_o, x)
        return (out, proj[:, at["out"]]) if self.gates_output else out


def distance_bucket(n: int, rows: int, far: float) -> int:
    """Row of a distance table of ``rows`` rows for a key ``n`` tokens back: exact in the first half, logarithmic up to ``far`` in
    the second."""
    half = rows // 2
    if n < half:
        return n
    if half == 0 or far <= half:
        return rows - 1
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def distance_table(rel, far: float, window: int):
    """(heads, n) fp32: the bias of a key d tokens back in column min(d, n - 1).  Columns end with the window or where the last
    bucket has been reached."""
    rows, idx = rel.shape[0], []
    for d in range(max(1, window)):
        idx.append(distance_bucket(d, rows, far))
        if idx[-1] == rows - 1:
            break
    return rel.float()[torch.tensor(idx, device=rel.device)].t().contiguous()


class RotaryTable:
    """cos and sin of position * frequency, rounded once from double precision: (2, positions, dims / 2) fp32.  One per rotation,
    shared by the layers that use it; the engine sizes it to its longest context.

    The frequencies are base^(-2 i / dims).  ``scaling`` with a ``factor`` alone divides all of them by it; with (factor, original, fast,
    slow) it interpolates them as YaRN does: pairs
    that turn more than ``fast`` times within ``original`` positions stay, those that turn less than ``slow`` times are slowed
    down by ``factor``, a linear ramp between; cos and sin are multiplied by 0.1 ln(factor) + 1."""

    def __init__(self, base: float, dims: int, device, scaling: dict | None = None):
        self.base, self.dims, self.device = float(base), int(dims), device
        self.table = None
        self.freq = self.base ** (-2.0 * torch.arange(self.dims // 2, dtype=torch.float64) / self.dims)
        self.gain = 1.0
        if scaling is not None and set(scaling) == {"factor"}:
            self.freq = self.freq / scaling["factor"]
        elif scaling is not None:
            pair = lambda turns: self.dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(self.base))
            lo, hi = max(math.floor(pair(scaling["fast"])), 0), min(math.ceil(pair(scaling["slow"])), self.dims - 1)
            ramp = ((torch.arange(self.dims // 2, dtype=torch.float64) - lo) / max(hi - lo, 0.001)).clamp(0.0, 1.0)
            self.freq = self.freq / scaling["factor"] * ramp + self.freq * (1.0 - ramp)
            self.gain = 0.1 * math.log(scaling["factor"]) + 1.0

    def resize(self, positions: int):
        if self.table is None or self.table.shape[1] != positions:
            angle = torch.outer(torch.arange(positions, dtype=torch.float64), self.freq)
            self.table = (self.gain * torch.stack((angle.cos(), angle.sin()))).float().contiguous().to(self.device)


class GatedFeedForward:
    """W_down (act(W_gate h) * (W_up h)), ``act`` "silu" or "relu"."""

    def __init__(self, get, width: int, ff: int, act: str, dtype, device, gain: float = 1.0):
        self.ff, self.act, self.gain = ff, act, float(gain)
        gu = torch.cat((_expect("gate", get("gate"), ff, width), _expect("up", get("up"), ff, width)))
        self.w_gu = mo.padded_weight(gu, dtype, device)                           # gate rows first
        self.w_down = mo.padded_weight(_expect("down", get("down"), width, ff), dtype, device)

    def __call__(self, h, x=None):
        return _project(mo.glu(h, self.w_gu, self.ff, self.act), self.w_down, x, self.gain)


class TableExperts:
    """SwiGLU experts chosen by a table row per token id, each with weight 1 / top; no router network.

    A step's rows are sorted by expert into 128-row tiles (``ops.mixer_ops.moe_plan``, once per step for all layers); the
    pass that norms a row also writes it where its experts read it, and the pass over the residual stream that follows
    adds the outputs up."""

    def __init__(self, get, width: int, ff: int, experts: int, top: int, vocab: int, dtype, device):
        self.ff, self.experts, self.top, self.width = ff, experts, top, width
        self.table = _expect("table", get("table"), vocab, top).to(device=device, dtype=torch.int32).contiguous()
        if int(self.table.min()) < 0 or int(self.table.max()) >= experts:
            raise ValueError("the expert table names an expert that does not exist")
        gu = torch.cat([_expect(f"e{e}.{k}", get(f"e{e}.{k}"), ff, width) for e in range(experts) for k in ("gate", "up")])
        self.w_gu = mo.padded_weight(gu, dtype, device)                            # (experts * 2 ff, width), gate first
        self.w_down = mo.padded_weight(torch.cat([_expect(f"e{e}.down", get(f"e{e}.down"), width, ff)
                                                  for e in range(experts)]), dtype, device)

    def rows(self, tokens: int) -> int:
        """Rows of the expert-sorted buffers for a step of ``tokens`` rows."""
        return mo.plan_tiles(tokens, self.experts, self.top) * mo.TILE

    def __call__(self, xg, tile_group):
        hidden = mo.gemm_rows(xg, self.w_gu, tile_group, self.ff, swiglu=True)
        return mo.gemm_rows(hidden, self.w_down, tile_group, self.width, swiglu=False)


class RoutedExperts:
    """Experts chosen by a learned router: W_down gelu(W_up h), or, ``gated``, W_down (silu(W_gate h) * (W_up h)).

    ``choice`` "logits": the ``top`` outputs with the largest logits (plus ``router.b``) are chosen, their weights are the softmax over the
    chosen logits.  "corrected": the router's softmax runs over ``experts`` + ``identity`` outputs; the last ``identity`` of them stand for h itself.  The ``top``
    outputs with the largest score + ``correction`` are chosen and weighted by their share of the chosen scores.  ``shared``: rows of
    an expert that every token uses, times sigmoid of one number per token (``shared.sg``, a row of the router's product).

    A step's rows are sorted by chosen expert into 128-row tiles for the grouped products; what comes out is added up by the next pass
    over the residual stream (``ops.mixer_ops.ExpertOutputs``).  In steps of few rows the shared expert is part of the grouped
    products too, if its rows are a multiple of the experts': in pieces of their size, which add up to it."""

    FOLD_ROWS = 256            # the largest step in which the shared expert joins the others

    def __init__(self, get, width: int, ff: int, experts: int, top: int, identity: int, shared: int | None, dtype, device,
                 gain: float = 1.0, gated: bool = False, choice: str = "corrected", out_gate=None):
        if not 0 < top <= experts + identity:
            raise ValueError(f"{top} of {experts + identity} outputs cannot be chosen")
        if choice not in ("corrected", "logits"):
            raise ValueError(f"unknown choice {choice!r}")
        if gated and shared is not None:
            raise ValueError("a shared expert is not gated")
        self.gated, self.gate = gated, None if out_gate is None else InputProducts({"out": out_gate[0]}, {"out": out_gate[1]}, dtype, device)
        self.width, self.ff, self.experts, self.top, self.identity, self.gain = width, ff, experts, top, identity, float(gain)
        w = lambda name, *shape: _expect(name, get(name), *shape)
        pack = lambda *ts: mo.padded_weight(torch.cat(ts), dtype, device)
        self.shared = shared is not None
        self.folds = shared // ff if self.shared and shared % ff == 0 else 0          # pieces of the shared expert among the others
        router = [w("router", experts + identity, width)]
        up = [w(f"e{e}.{k}", ff, width) for e in range(experts) for k in (("gate", "up") if gated else ("up",))]
        down = [w(f"e{e}.down", width, ff) for e in range(experts)]
        if self.shared:
            router.append(w("shared.sg", 1, width))
            s_up, s_down = w("shared.up", shared, width), w("shared.down", width, shared)
            up += list(s_up.split(ff)) if self.folds else []
            down += list(s_down.split(ff, 1)) if self.folds else []
        self.w_router, self.w_up, self.w_down = pack(*router), pack(*up), pack(*down)
        if self.shared:
            self.w_shared_up = self.w_up[experts * ff:] if self.folds else pack(s_up)
            self.w_shared_down = self.w_down[experts * width:] if self.folds == 1 else pack(s_down)
        f32 = lambda name: w(name, experts + identity).to(device=device, dtype=torch.float32).contiguous()
        self.correction, self.bias = (f32("correction"), None) if choice == "corrected" else (None, f32("router.b"))

    def __call__(self, h, slots, count):
        """``count``: (experts,) int32 of zeros."""
        outputs, rows = self.experts + self.identity, h.shape[0]
        fold = self.folds if rows <= self.FOLD_ROWS else 0
        cols = outputs + (fold > 0)
        if mo.routes_rows(rows, self.w_router):
            z, choice, rank, weight = mo.moe_route_rows(h, self.w_router, self.correction, slots, self.experts, self.top, count, fold,
                                                        self.bias)
        else:
            z = mo.linear(h, self.w_router, out_dtype=torch.float32)               # what is routed by is 32-bit
            choice, rank, weight = mo.moe_route(z[:, :cols], self.correction, slots, self.experts, self.top, count, fold, self.bias)
        xg, pos, groups = mo.moe_dispatch(h, choice, rank, count, fold)
        y = mo.gemm_rows(mo.gemm_rows(xg, self.w_up, groups, self.ff, self.gated, None if self.gated else "gelu"), self.w_down, groups, self.width,
                         False)
        if self.gate is not None:
            return mo.ExpertOutputs(y, pos, self.gain, weight, h if self.identity else None), self.gate(h)[:, self.gate.at["out"]]
        if fold or not self.shared:
            return mo.ExpertOutputs(y, pos, self.gain, weight, h)
        s = mo.linear(mo.linear(h, self.w_shared_up, act="gelu"), self.w_shared_down)
        return mo.ExpertOutputs(y, pos, self.gain, weight, h, s, z[:, outputs])
