"""What the serving engine needs from a model: its cache, one step of its layers, its logits.

``ServingEngine`` owns requests, pages, slots, batches, graphs and sampling; a backend runs the layers of one
``StepBatch``.  ``forward`` returns whatever ``logits`` takes; both run inside CUDA-graph capture when the batch has no
portions.  ``splits_prompts`` says whether a long prompt is fed in several portions (its backend reads the earlier ones
from the cache efficiently)."""
from __future__ import annotations

import numpy as np
import torch

from .. import ops
from ..ops import mixer_ops as mo
from ..ops import serving_ops
from .kv_cache import LayerCache, PagedKVCache, StateSpec


class TransformerBackend:
    """``TransformerLM``: packed QKV attention with rotary pairs, K and V pages, bf16 residual stream."""

    splits_prompts = False
    page_size = 16

    def __init__(self, model):
        model.use_custom_triton = True
        eng = model.engine()
        prov = eng.provider
        prov.begin_step()                       # builds the bf16 weight mirror and its views
        self.cfg = eng.cfg
        self.layers = [prov.block_weights(i) for i in range(self.cfg.n_layers)]
        self.head = prov.head_weights()
        self.rope = eng.rope_cache
        self.device = self.head.emb.device
        self.dtype = self.head.emb.dtype
        self.vocab = self.cfg.vocab
        self.context_limit = min(model.context_length, self.rope.shape[1])
        self.default_context = self.context_limit

    def set_context(self, positions: int):
        pass

    def page_bytes(self, page_size: int) -> int:
        return PagedKVCache.bytes_per_page(self.cfg.n_layers, self.cfg.d_model, page_size,
                                           2 if self.dtype == torch.bfloat16 else 4)

    def make_cache(self, num_pages: int, page_size: int, max_batch: int):
        self.cache = PagedKVCache(self.cfg.n_layers, self.cfg.d_model, num_pages, page_size, self.device, self.dtype)
        return self.cache

    def choose_splits(self, rows: int, max_context: int) -> int:
        return serving_ops.choose_splits(rows, self.cfg.n_heads, max_context, head_dim=self.cfg.d_model // self.cfg.n_heads)

    def _block(self, x, w, li: int, batch, attend):
        cfg = self.cfg
        h, _ = ops.rmsnorm_fwd(x, w.n1, cfg.eps)
        qkv = ops.gemm(h, w.wqkv, "nt", b_stable=True)
        # rotary embedding of Q and K in place and the append of K, V to the paged cache: one kernel on the GPU
        serving_ops.rope_kv_append(qkv, self.rope, batch.positions, self.cache.k[li], self.cache.v[li], batch.slots, cfg.n_heads)
        o = attend(qkv, li)
        x = ops.gemm(o, w.wo, "nt", residual=x, b_stable=True)
        h, _ = ops.rmsnorm_fwd(x, w.n2, cfg.eps)
        gu = ops.gemm(h, w.wgu, "nt", b_stable=True)
        return ops.gemm(ops.silu_mul_fwd(gu), w.wdown, "nt", residual=x, b_stable=True)

    def forward(self, batch):
        heads = self.cfg.n_heads
        if batch.n_single == batch.n_rows:
            tables, ctx = batch.tables, batch.ctx
        elif batch.n_single == 0 and all(start == 0 for start, _ in batch.portions):
            tables = None
        else:
            # portions that continue a prompt, or portions beside single tokens: every row attends to its own request's
            # pages up to its position, as a decode step does (its K and V are in the cache by then)
            tables, ctx = batch.tables[batch.row_seq.long()], batch.positions + 1

        def attend(qkv, li):
            if tables is not None:
                return serving_ops.paged_decode_attention(qkv, self.cache.k[li], self.cache.v[li], tables, ctx, heads,
                                                          batch.splits)
            if qkv.is_cuda:
                from ..ops import attention
                return attention.varlen_attention_fwd(qkv, batch.cu, batch.max_portion, heads)
            return ops.torch_impl.varlen_attention_fwd(qkv, batch.cu, heads)

        x = ops.embedding_fwd(batch.tokens, self.head.emb)
        for li, w in enumerate(self.layers):
            x = self._block(x, w, li, batch, attend)
        return x

    def logits(self, x, rows=None):
        """(rows, padded vocabulary): only the first ``vocab`` columns are defined."""
        if rows is not None:
            x = x[rows].contiguous()
        h, _ = ops.rmsnorm_fwd(x, self.head.norm, self.cfg.eps)
        buf = torch.empty((x.shape[0], self.cfg.vocab_padded), dtype=x.dtype, device=x.device)
        ops.gemm(h, self.head.lm, "nt", out=buf[:, :self.cfg.vocab], b_stable=True)
        return buf


class LayeredBackend:
    """What models made of listed layers (``models/layered.py``) have in common: one cache entry per layer run, an fp32
    residual stream, fp32 logits.  A subclass knows the order of a layer's sublayers and norms."""

    splits_prompts = True
    page_size = 64                    # tokens: the attention kernels copy whole pages as TMA boxes

    def __init__(self, model):
        self.model = model
        self.device, self.dtype, self.vocab = model.device, model.dtype, model.vocab_size
        self.context_limit = None
        self.default_context = model.DEFAULT_CONTEXT
        self.specs = [layer.mixer.cache_spec() for layer in model.runs]

    def set_context(self, positions: int):
        for table in self.model.rotary.values():
            table.resize(positions)

    def page_bytes(self, page_size: int) -> int:
        return LayerCache.bytes_per_page(self.specs, page_size, self.dtype.itemsize)

    def make_cache(self, num_pages: int, page_size: int, max_batch: int):
        self.cache = LayerCache(self.specs, num_pages, page_size, max_batch, self.device, self.dtype)
        return self.cache

    def choose_splits(self, rows: int, max_context: int) -> int:
        return 0

    def stream(self, batch):
        """The residual stream of a step, not yet written."""
        batch.gathered.clear()
        return torch.empty((batch.n_rows, self.model.config.width), dtype=torch.float32, device=self.device)

    def head(self, h, cap: float | None = None, scale: float = 1.0):
        """(rows, vocabulary) fp32 of normed rows, times ``scale``; ``cap``: capped softly."""
        out = torch.empty((h.shape[0], mo.pitch(self.vocab)), dtype=torch.float32, device=self.device)
        mo.linear(h, self.model.head, out=out[:, :self.vocab], alpha=scale, act="cap" if cap else None, cap=cap or 0.0)
        return out


class ParallelLayers(LayeredBackend):
    """Parallel sublayers on one norm, token-table experts (``models/tedirax.py``).

    A layer run is: one pass over the residual stream (add the previous run's expert outputs, norm, copy rows to where
    the experts read them), the mixer (adds to the residual stream in its last product), the experts."""

    def __init__(self, model):
        super().__init__(model)
        self.expert_layers = [layer for layer in model.layers if layer.experts is not None]

    def forward(self, batch, trace=None):
        """``trace``: a list that receives the residual stream after every layer run (a copy; for tests)."""
        m = self.model
        x = self.stream(batch)
        plan = {}
        if self.expert_layers:
            pos, groups = mo.moe_plan(batch.tokens, batch.slots, [la.experts.table for la in self.expert_layers],
                                      [la.experts.experts for la in self.expert_layers])
            plan = {la.index: (p, g) for la, p, g in zip(self.expert_layers, pos, groups)}
        embed, pending = (batch.tokens, m.embed), None
        for run, layer in enumerate(m.runs):
            ex = layer.experts
            scatter = None
            if ex is not None:
                pos, groups = plan[layer.index]
                scatter = (pos, ex.rows(batch.n_rows))
            h, xg = mo.residual_norm(x, layer.norm, m.config.eps, tokens=embed[0], embed=embed[1], pending=pending,
                                     scatter=scatter)
            embed, pending = (None, None), None
            layer.mixer(h, x, batch, self.cache.entries[run])
            if ex is not None:
                pending = (ex(xg, groups), pos, 1.0 / ex.top)
            if trace is not None:
                if pending is not None:
                    mo.residual_norm(x, pending=pending)
                    pending = None
                trace.append(x.clone())
        if not m.runs:
            mo.residual_norm(x, tokens=batch.tokens, embed=m.embed)
        return x, pending

    def logits(self, hidden, rows=None):
        """(rows, vocabulary) fp32."""
        x, pending = hidden
        m = self.model
        if rows is None:
            h, _ = mo.residual_norm(x, m.final_norm, m.config.eps, pending=pending)
        else:
            h, _ = mo.residual_norm(x, m.final_norm, m.config.eps, row_index=rows, pending=pending)
        return self.head(h)


class PostNormLayers(LayeredBackend):
    """Sublayers one after the other, each reading the residual stream itself, its output normed before it is added
    (``models/beledra.py``).  The pass that adds a sublayer's output also writes the next one's input."""

    def forward(self, batch, trace=None):
        """``trace``: a list that receives the residual stream after every layer run (a copy; for tests)."""
        m, eps = self.model, self.model.config.eps
        x = self.stream(batch)
        h = mo.add_normed(x, tokens=batch.tokens, embed=m.embed)
        for run, layer in enumerate(m.runs):
            h = mo.add_normed(x, layer.mixer(h, None, batch, self.cache.entries[run]), layer.norm1, eps)
            if layer.mlp is not None:
                h = mo.add_normed(x, layer.mlp(h), layer.norm2, eps)
            if trace is not None:
                trace.append(x.clone())
        return x

    def logits(self, x, rows=None):
        """(rows, vocabulary) fp32."""
        h, _ = mo.residual_norm(x, self.model.final_norm, self.model.config.eps, row_index=rows)
        return self.head(h)


class PreNormLayers(LayeredBackend):
    """Sublayers one after the other, each reading a norm of the residual stream and adding its output times a gain
    (``models/genedra.py``).  Products add into the stream in their epilogues; the outputs of experts are added by the pass that
    makes the next sublayer's input."""

    def __init__(self, model):
        super().__init__(model)
        self.counters = [layer.mlp.experts for layer in model.layers if layer.routed]

    def forward(self, batch, trace=None):
        """``trace``: a list that receives the residual stream after every layer run (a copy; for tests)."""
        m, cfg = self.model, self.model.config
        x = self.stream(batch)
        counts = None
        if self.counters:
            counts = iter(torch.zeros(sum(self.counters), dtype=torch.int32, device=self.device).split(self.counters))
        start = dict(tokens=batch.tokens, embed=m.embed, embed_scale=cfg.embed_scale)
        pending = None
        for run, layer in enumerate(m.runs):
            h, _ = mo.residual_norm(x, layer.norm1, cfg.eps, pending=pending, w_offset=1.0, **start)
            start, pending = {}, None
            layer.mixer(h, x, batch, self.cache.entries[run])
            if layer.mlp is not None:
                h, _ = mo.residual_norm(x, layer.norm2, cfg.eps, w_offset=1.0)
                if layer.routed:
                    pending = layer.mlp(h, batch.slots, next(counts))
                else:
                    layer.mlp(h, x)
            if trace is not None:
                if pending is not None:
                    mo.residual_norm(x, pending=pending)
                    pending = None
                trace.append(x.clone())
        if start:
            mo.residual_norm(x, **start)
        return x, pending

    def logits(self, hidden, rows=None):
        """(rows, vocabulary) fp32."""
        x, pending = hidden
        m = self.model
        h, _ = mo.residual_norm(x, m.final_norm, m.config.eps, row_index=rows, pending=pending, w_offset=1.0)
        return self.head(h, m.config.logit_softcap)


class SandwichLayers(LayeredBackend):
    """Sublayers one after the other, each reading a group norm of the residual stream; its output is multiplied by a gate of the same input
    and normed before it is added (``models/vilosun.py``).  The pass that adds a sublayer's output also writes the next one's input; the last
    one belongs to the logits.  The embedding of token pairs keeps every request's last token in its state slot."""

    def __init__(self, model):
        super().__init__(model)
        self.counters = [layer.mlp.experts for layer in model.layers if layer.mlp is not None]
        self.specs = [*self.specs, StateSpec((1,), "tokens")]

    def forward(self, batch, trace=None):
        """``trace``: a list that receives the residual stream after every layer run (a copy; for tests)."""
        m, cfg = self.model, self.model.config
        x = self.stream(batch)
        counts = None
        if self.counters:
            counts = iter(torch.zeros(sum(self.counters), dtype=torch.int32, device=self.device).split(self.counters))
        step = lambda w, **kw: mo.group_step(x, cfg.groups, cfg.eps, w, **kw)
        start = mo.EmbeddingStart(m.embed, cfg.embed_scale, m.bigram, cfg.mul_prev, cfg.mul_cur, self.cache.entries[-1])
        h, pending = step(m.runs[0].norm1 if m.runs else None, start=start, batch=batch), None
        for run, layer in enumerate(m.runs):
            if pending is not None:
                h = step(layer.norm1, sub=pending)
            pending = mo.GatedOutput(*layer.mixer(h, None, batch, self.cache.entries[run]), layer.norm1b)
            if layer.mlp is not None:
                h = step(layer.norm2, sub=pending)
                pending = mo.GatedOutput(*layer.mlp(h, batch.slots, next(counts)), layer.norm2b)
            if trace is not None:
                after = m.runs[run + 1].norm1 if run + 1 < len(m.runs) else None
                h, pending = step(after, sub=pending), None
                trace.append(x.clone())
        return x, pending

    def logits(self, hidden, rows=None):
        """(rows, vocabulary) fp32."""
        x, pending = hidden
        cfg = self.model.config
        h = mo.group_step(x, cfg.groups, cfg.eps, self.model.final_norm, sub=pending, row_index=rows)
        return self.head(h, scale=cfg.logit_scale)


def wanted_index(rows: np.ndarray, device) -> torch.Tensor:
    t = torch.from_numpy(np.ascontiguousarray(rows, dtype=np.int64))
    return t.pin_memory().to(device, non_blocking=True) if torch.device(device).type == "cuda" else t
