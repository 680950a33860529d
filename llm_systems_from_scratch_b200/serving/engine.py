"""Continuous-batching inference engine over a paged cache (and recurrent state slots, for models that have them).

New capability relative to the reference, whose only inference path is ``TransformerLM.generate``
(batch 1, no KV cache, llm-core/llm_core/model.py:187-236).  One engine instance drives one GPU;
data-parallel serving runs one replica process per GPU.

Per iteration: newly admitted prompts are packed into one variable-length step whose keys and states go straight
into the cache (models that can continue a prompt get long ones in portions of at most ``max_prefill_tokens``), then
every running request advances by one token in a single decode step.  Decode steps are captured in
CUDA graphs, one per padded batch-size bucket, because at a few milliseconds per step the ~250 kernel
launches of a step would otherwise be launch bound.  Greedy sampling runs on the device.

The layers belong to the model's backend (``serving.backends``): the engine hands it one ``StepBatch`` at a time,
whether that is a prompt, a decode step or - ``extend``, for callers that bring the tokens themselves - any mixture.
"""
from __future__ import annotations

import gc
import time

import numpy as np
import torch

from .. import ops
from ..utils.metrics import Percentiles
from .backends import wanted_index
from .batch import StepBatch
from .scheduler import Request, Scheduler


class ServingEngine:
    BUCKETS = (1, 2, 4, 8, 16, 32, 64, 128, 256)

    def __init__(self, model, num_pages: int | None = None, page_size: int | None = None, max_batch: int = 64,
                 max_context: int | None = None, max_prefill_tokens: int = 8192, use_cuda_graphs: bool = True,
                 kv_memory_fraction: float = 0.5):
        self.backend = be = model.serving_backend()
        self.device, self.dtype = be.device, be.dtype
        self.cuda = self.device.type == "cuda"
        self.max_context = max_context or be.default_context
        if be.context_limit is not None:
            self.max_context = min(self.max_context, be.context_limit)
        be.set_context(self.max_context)
        self.page_size = page_size = page_size or be.page_size
        self.max_pages_per_req = -(-self.max_context // page_size)
        if num_pages is None:
            per_page = be.page_bytes(page_size)
            if self.cuda and per_page:
                free, _ = torch.cuda.mem_get_info(self.device)
                num_pages = max(self.max_pages_per_req * 2, int(free * kv_memory_fraction) // per_page)
                num_pages = min(num_pages, self.max_pages_per_req * max_batch + 8)
            else:
                num_pages = self.max_pages_per_req * max_batch
        self.cache = be.make_cache(num_pages, page_size, max_batch)
        self.sched = Scheduler(self.cache.allocator, page_size, max_batch, max_prefill_tokens, self.max_context,
                               self.cache.slot_allocator)
        self._prefilling: list[Request] = []        # admitted, prompt not yet fed completely
        self.max_batch = max_batch
        self.use_graphs = use_cuda_graphs and self.cuda
        self._graphs: dict[int, dict] = {}
        try:
            from ..utils import host_runtime
            self._host_rt = host_runtime if host_runtime.available() else None
        except Exception:
            self._host_rt = None
        self._temperature, self._top_k = 0.0, None
        self.stats = {"prefill_tokens": 0, "decode_tokens": 0, "decode_steps": 0, "prefill_steps": 0}

    # ----------------------------------------------------------------------- sampling
    def _greedy(self, logits_buf):
        """Next token per row: argmax, or a draw from softmax(logits / temperature) over the top-k logits when
        ``set_sampling`` asked for one (one kernel on the GPU: filter, softmax and inverse-CDF draw, no sort)."""
        if self._temperature == 0:
            return ops.argmax_rows(logits_buf, self.backend.vocab)
        rows = logits_buf.shape[0]
        if logits_buf.is_cuda:
            u = torch.rand(rows, device=logits_buf.device)
            return ops.sample_topk(logits_buf, u, self._temperature, self._top_k, self.backend.vocab)
        last = logits_buf[:, :self.backend.vocab].float() / self._temperature
        if self._top_k:
            kth = torch.topk(last, min(self._top_k, last.shape[-1])).values[:, -1:]
            last = last.masked_fill(last < kth, float("-inf"))
        return torch.multinomial(torch.softmax(last, dim=-1), 1).reshape(-1)

    def set_sampling(self, temperature: float = 0.0, top_k: int | None = None):
        """temperature 0 = greedy.  Decode graphs captured under another setting are dropped."""
        if (temperature, top_k) != (self._temperature, self._top_k):
            self._temperature, self._top_k = float(temperature), top_k
            self._graphs.clear()

    # ------------------------------------------------------------------------ prefill
    def _run_portions(self, work: list[tuple[Request, int]]) -> torch.Tensor:
        """Feed the next ``n`` prompt tokens of every (request, n); returns the token sampled behind each portion."""
        batch = StepBatch.build([(r, r.fed, r.prompt[r.fed:r.fed + n]) for r, n in work], self.page_size,
                                self.max_pages_per_req, self.device)
        hidden = self.backend.forward(batch)
        first = self._greedy(self.backend.logits(hidden, wanted_index(batch.last_rows(), self.device)))
        for r, n in work:
            r.fed += n
        self.stats["prefill_tokens"] += sum(n for _, n in work)
        self.stats["prefill_steps"] += 1
        return first

    @torch.no_grad()
    def prefill(self, reqs: list[Request]) -> torch.Tensor:
        """Run the prompts of ``reqs`` (pages already reserved) in one step; returns their first generated tokens."""
        return self._run_portions([(r, len(r.prompt) - r.fed) for r in reqs])

    # ------------------------------------------------------------- tokens brought by the caller
    def open(self, rid) -> Request:
        """A request whose tokens the caller brings step by step (``extend``) until ``close``."""
        req = Request(rid, [], 0)
        self.sched.open(req)
        return req

    def close(self, req: Request):
        self.sched.finish(req)

    @torch.no_grad()
    def extend(self, entries: list[tuple[Request, list[int], list[int]]]) -> torch.Tensor | None:
        """Run one step that brings (request, its next tokens, places among them whose logits are wanted) for every
        entry, all as one batch: single tokens beside portions of any length.  Returns the logits of the wanted places,
        entry by entry, (wanted, vocabulary) fp32, or None when nothing is wanted."""
        for r, ids, _ in entries:
            if not ids:
                raise ValueError(f"request {r.rid} brings no token")
            self.sched.grow(r, r.fed + len(ids))
        if not entries:
            return None
        batch = StepBatch.build([(r, r.fed, ids) for r, ids, _ in entries], self.page_size, self.max_pages_per_req,
                                self.device)
        hidden = self.backend.forward(batch)
        for r, ids, _ in entries:
            r.fed += len(ids)
        rows = batch.wanted_rows([want for _, _, want in entries])
        if not len(rows):
            return None
        return self.backend.logits(hidden, wanted_index(rows, self.device))[:, :self.backend.vocab].float()

    # ------------------------------------------------------------------------- decode
    def _decode_body(self, d: dict, n: int, splits: int):
        """One decode step of the first ``n`` rows of the device arrays ``d``; returns their next tokens."""
        batch = StepBatch(d["tokens"][:n], d["positions"][:n], d["slots"][:n], d["tables"][:n], d["ctx"][:n],
                          d["state"][:n], d["rows"][:n], n, splits=splits)
        return self._greedy(self.backend.logits(self.backend.forward(batch)))

    def _arrays(self, n: int) -> dict:
        """Device arrays of a decode step of ``n`` rows, all rows idle."""
        dev = self.device
        return {"tokens": torch.zeros(n, dtype=torch.int64, device=dev),
                "positions": torch.zeros(n, dtype=torch.int32, device=dev),
                "slots": torch.full((n,), -1, dtype=torch.int64, device=dev),
                "ctx": torch.ones(n, dtype=torch.int32, device=dev),
                "state": torch.full((n,), -1, dtype=torch.int32, device=dev),
                "rows": torch.arange(n, dtype=torch.int32, device=dev),
                "tables": torch.zeros((n, self.max_pages_per_req), dtype=torch.int32, device=dev)}

    def _capture(self, d: dict, n: int, run) -> torch.cuda.CUDAGraph:
        """Capture ``run`` (a decode step of the first n rows of ``d``).  The warm-up run before it, where first-launch
        set-up happens, sees idle rows only: a recurrent state must not advance twice."""
        keep = {k: d[k][:n].clone() for k in ("tokens", "slots", "state")}
        d["slots"][:n] = -1
        d["state"][:n] = -1
        side = torch.cuda.Stream(device=self.device)
        side.wait_stream(torch.cuda.current_stream())
        with torch.cuda.stream(side):
            run()
        torch.cuda.current_stream().wait_stream(side)
        torch.cuda.synchronize()
        graph = torch.cuda.CUDAGraph()
        # an engine that is no longer used would take its graphs with it when the collector finds it, which a capture does not survive
        gc.collect()
        collects = gc.isenabled()
        gc.disable()
        try:
            with torch.cuda.graph(graph):
                run()
        finally:
            if collects:
                gc.enable()
        for k, v in keep.items():
            d[k][:n].copy_(v)
        return graph

    def _bucket(self, n: int) -> int:
        for b in self.BUCKETS:
            if b >= n:
                return b
        return n

    def _graph_for(self, bucket: int) -> dict:
        g = self._graphs.get(bucket)
        if g is not None:
            return g
        st = self._arrays(bucket)
        splits = self.backend.choose_splits(bucket, self.max_context)
        st["out"] = torch.zeros(bucket, dtype=torch.int64, device=self.device)

        def run():
            st["out"].copy_(self._decode_body(st, bucket, splits))
        if self.use_graphs:
            st["graph"] = self._capture(st, bucket, run)
        st["run"] = run
        st["splits"] = splits
        self._graphs[bucket] = st
        return st

    @torch.no_grad()
    def decode(self, reqs: list[Request]) -> list[int]:
        """Advance every request in ``reqs`` by one token; returns the new tokens (host ints)."""
        n = len(reqs)
        bucket = self._bucket(n)
        st = self._graph_for(bucket)
        ps = self.page_size
        # Host staging is pinned once per bucket and refilled in place through numpy views (the previous step ended
        # with a device-to-host read, so no copy from these buffers is still in flight).
        host = st.get("host")
        if host is None:
            mk = lambda shape, dt: torch.zeros(shape, dtype=dt, pin_memory=self.cuda)
            host = st["host"] = {"tokens": mk(bucket, torch.int64), "positions": mk(bucket, torch.int32),
                                 "slots": mk(bucket, torch.int64), "ctx": mk(bucket, torch.int32),
                                 "state": mk(bucket, torch.int32),
                                 "tables": mk((bucket, self.max_pages_per_req), torch.int32)}
            st["host_np"] = {k: v.numpy() for k, v in host.items()}
        hn = st["host_np"]
        p = np.fromiter((r.context_len - 1 for r in reqs), dtype=np.int64, count=n)   # position of the token being fed
        hn["tokens"][:n] = np.fromiter((r.output[-1] for r in reqs), dtype=np.int64, count=n)
        hn["tokens"][n:] = 0
        hn["positions"][:n] = p
        hn["positions"][n:] = 0
        hn["slots"][:n] = np.fromiter((r.pages[q // ps] for r, q in zip(reqs, p)), dtype=np.int64, count=n) * ps + p % ps
        hn["slots"][n:] = -1
        hn["ctx"][:n] = p + 1
        hn["ctx"][n:] = 1
        hn["state"][:n] = [r.slot for r in reqs]
        hn["state"][n:] = -1
        if self._host_rt is not None:
            self._host_rt.block_table_into([r.pages for r in reqs], host["tables"], 0)
        else:
            tb = hn["tables"]
            tb[:] = 0
            for i, r in enumerate(reqs):
                tb[i, :len(r.pages)] = r.pages
        for name in ("tokens", "positions", "slots", "ctx", "state", "tables"):
            st[name].copy_(host[name], non_blocking=True)
        if self.use_graphs:
            st["graph"].replay()
        else:
            st["run"]()
        new = st["out"][:n].tolist()
        self.stats["decode_tokens"] += n
        self.stats["decode_steps"] += 1
        return new

    # ---------------------------------------------------------------------- main loop
    # Requests keep one row of the batch arrays for their whole life; the token each row feeds next stays on the
    # device (the decode graph copies its output there), so a decode step can be launched before the previous step's
    # tokens have reached the host.  The host reads them one step behind: while step k + 1 runs on the GPU it appends
    # step k's tokens, retires finished requests and prepares step k + 2.
    def _rows_init(self):
        n = self._bucket(self.max_batch)
        self._row_req: list[Request | None] = [None] * n
        self._row_pos = np.full(n, -1, dtype=np.int64)        # position of the token the row feeds next; -1 = idle
        self._row_tab = np.zeros((n, self.max_pages_per_req), dtype=np.int64)
        self._free_rows = list(range(n - 1, -1, -1))
        self._d = self._arrays(n)
        mk = lambda shape, dt: torch.zeros(shape, dtype=dt, pin_memory=self.cuda)
        # two sets of pinned staging used in turn: a set is refilled only after the step before last has completed
        self._stage = [{"positions": mk(n, torch.int32), "slots": mk(n, torch.int64), "ctx": mk(n, torch.int32),
                        "state": mk(n, torch.int32), "out": mk(n, torch.int64)} for _ in range(2)]
        self._stage_np = [{k: v.numpy() for k, v in st.items()} for st in self._stage]
        self._tab_host = mk((n, self.max_pages_per_req), torch.int32)
        self._state_host = mk(n, torch.int32)
        self._state_host.fill_(-1)
        self._tab_dirty = False
        self._parity = 0
        self._pending: list[tuple] = []
        self._row_graphs: dict[int, dict] = {}

    def _row_graph(self, bucket: int) -> dict:
        g = self._row_graphs.get(bucket)
        if g is not None:
            return g
        d = self._d
        splits = self.backend.choose_splits(bucket, self.max_context)

        def run():
            out = self._decode_body(d, bucket, splits)
            d["tokens"][:bucket].copy_(out)          # the next step of every row starts from this token
        g = {"run": run}
        if self.use_graphs:
            g["graph"] = self._capture(d, bucket, run)
        self._row_graphs[bucket] = g
        return g

    def warmup(self):
        """Capture the decode graph of every batch bucket up to ``max_batch`` now, so that no request of a trace pays
        for a capture (a few tenths of a second each) with its time to first token."""
        if not hasattr(self, "_row_req"):
            self._rows_init()
        if self.use_graphs:
            top = self._bucket(self.max_batch)
            for b in self.BUCKETS:
                if b <= top:
                    self._row_graph(b)
            torch.cuda.synchronize()

    def _admit_rows(self, reqs: list[Request], first: torch.Tensor):
        rows = [self._free_rows.pop() for _ in reqs]
        for row, r in zip(rows, reqs):
            self._row_req[row] = r
            r.row = row
            r.issued = 1                                     # the prefill produced the first token
            self._row_pos[row] = len(r.prompt)
            self._row_tab[row, :] = 0
            self._row_tab[row, :len(r.pages)] = r.pages
            if r.issued >= r.max_new_tokens:
                self._row_pos[row] = -1                      # nothing left to decode
        self._tab_host.numpy()[rows] = self._row_tab[rows]
        self._state_host.numpy()[rows] = [r.slot for r in reqs]
        self._tab_dirty = True
        idx = torch.tensor(rows, dtype=torch.int64)
        if self.cuda:
            idx = idx.pin_memory().to(self.device, non_blocking=True)
        self._d["tokens"].index_copy_(0, idx, first.to(torch.int64))
        self._read_back("prefill", first, list(zip(range(len(reqs)), reqs)))

    def _read_back(self, kind: str, dev_tokens: torch.Tensor, who: list):
        """Queue a device-to-host read of ``dev_tokens``; ``who`` lists (index into it, request)."""
        if self.cuda:
            host = torch.empty(dev_tokens.shape, dtype=torch.int64, pin_memory=True) if kind == "prefill" else \
                self._stage[self._parity]["out"][:dev_tokens.shape[0]]
            host.copy_(dev_tokens, non_blocking=True)
            ev = torch.cuda.Event()
            ev.record()
        else:
            host, ev = dev_tokens.clone(), None
        self._pending.append((kind, ev, host, who))

    def _launch_decode(self) -> int:
        active = np.nonzero(self._row_pos >= 0)[0]
        if active.size == 0:
            return 0
        bucket = self._bucket(int(active[-1]) + 1)
        ps = self.page_size
        st = self._stage_np[self._parity]
        pos = self._row_pos[:bucket]
        live = pos >= 0
        p = np.where(live, pos, 0)
        st["positions"][:bucket] = p
        st["slots"][:bucket] = np.where(live, self._row_tab[np.arange(bucket), p // ps] * ps + p % ps, -1)
        st["ctx"][:bucket] = np.where(live, p + 1, 1)
        d, host = self._d, self._stage[self._parity]
        for name in ("positions", "slots", "ctx"):
            d[name][:bucket].copy_(host[name][:bucket], non_blocking=True)
        if self._tab_dirty:
            d["tables"].copy_(self._tab_host, non_blocking=True)
            self._tab_dirty = False
        # an idle row must not touch a state: its slot may belong to another request by now
        st["state"][:bucket] = np.where(live, self._state_host.numpy()[:bucket], -1)
        d["state"][:bucket].copy_(host["state"][:bucket], non_blocking=True)
        g = self._row_graph(bucket)
        if self.use_graphs:
            g["graph"].replay()
        else:
            g["run"]()
        who = [(int(row), self._row_req[row]) for row in active]
        self._read_back("decode", d["tokens"][:bucket], who)
        self._parity ^= 1
        # bookkeeping that needs no token values: positions advance, rows whose last token is now in flight go idle
        self._row_pos[active] += 1
        for row, r in who:
            r.issued += 1
            if r.issued >= r.max_new_tokens:
                self._row_pos[row] = -1
        self.stats["decode_tokens"] += len(who)
        self.stats["decode_steps"] += 1
        return len(who)

    def _finish(self, keep_last: int = 0) -> int:
        """Consume queued read-backs, oldest first, leaving the ``keep_last`` most recent ones in flight."""
        produced = 0
        while len(self._pending) > keep_last:
            kind, ev, host, who = self._pending.pop(0)
            if ev is not None:
                ev.synchronize()
            vals = host.numpy() if host.device.type == "cpu" else host.cpu().numpy()
            t = self._clock()
            for i, r in who:
                if r.t_done is not None:
                    continue                                  # ended by its stop token a step earlier
                r.output.append(int(vals[i]))
                produced += 1
                if kind == "prefill":
                    r.t_first = t
                if r.finished:
                    r.t_done = t
                    row = r.row
                    self._row_pos[row] = -1
                    self._row_req[row] = None
                    self._free_rows.append(row)
                    self.sched.finish(r)
        return produced

    def cancel(self, req: Request) -> bool:
        """Stop ``req`` now: a waiting request leaves the queue, a running one gives its row and its KV pages back and
        keeps the tokens that have reached the host.  Like a stop token, it may have one decode step in flight; that
        step's token is dropped when it is read, and its KV write lands (in stream order) before anything a later owner
        of the pages writes.  Returns False if the request had already finished."""
        if req.t_done is not None:
            return False
        if req in self.sched.waiting:
            self.sched.waiting.remove(req)
            req.t_done = self._clock()
            return True
        if req in self._prefilling:
            self._prefilling.remove(req)
            req.t_done = self._clock()
            self.sched.finish(req)
            return True
        if req.row < 0 or self._row_req[req.row] is not req:
            return False
        row = req.row
        req.t_done = self._clock()
        self._row_pos[row] = -1
        self._row_req[row] = None
        self._free_rows.append(row)
        self.sched.finish(req)
        return True

    def step(self, now: float) -> int:
        """One engine iteration at time ``now``: admit + prefill, launch one decode step, then collect the tokens
        of the step before.  Returns the number of tokens that reached the host."""
        if not hasattr(self, "_row_req"):
            self._rows_init()
        admitted = self.sched.admit(now)
        if admitted:
            self.sched.start(admitted)
            self._prefilling.extend(admitted)
        if self._prefilling:
            self._prefill_step()
        launched = self._launch_decode()
        # on the GPU the newest read-back stays in flight while the host goes on; when nothing was launched (every
        # row's last token is already in flight) or without streams, everything is collected now
        return self._finish(keep_last=1 if (self.cuda and launched) else 0)

    @torch.no_grad()
    def _prefill_step(self):
        """Feed prompts, oldest request first, up to the token budget of a step; requests whose prompt is complete join
        the decode rows.  Without portions every prompt goes whole (admission kept their sum to the budget)."""
        budget, work = self.sched.max_prefill_tokens, []
        for r in self._prefilling:
            n = len(r.prompt) - r.fed
            if self.backend.splits_prompts:
                n = min(n, budget)
                if n <= 0:
                    break
                budget -= n
            work.append((r, n))
        first = self._run_portions(work)
        done = [i for i, (r, _) in enumerate(work) if r.fed == len(r.prompt)]
        if not done:
            return
        ready = [work[i][0] for i in done]
        self._prefilling = [r for r in self._prefilling if r.fed < len(r.prompt)]
        if len(done) < len(work):
            first = first[wanted_index(np.asarray(done), self.device)]
        self._admit_rows(ready, first)

    def _clock(self) -> float:
        return time.perf_counter() - self._t0 if self._realtime else self._virtual

    def run(self, requests: list[Request], realtime: bool = True) -> dict:
        """Replay ``requests`` (sorted by arrival).  ``realtime`` honours arrival times against the wall
        clock; otherwise every request counts as already arrived (offline throughput)."""
        self._realtime = realtime
        self._virtual = float("inf")
        for r in sorted(requests, key=lambda q: q.arrival):
            self.sched.add(r)
        if self.cuda:
            torch.cuda.synchronize()
        self._t0 = time.perf_counter()
        if not hasattr(self, "_row_req"):
            self._rows_init()
        while not self.sched.idle or self._pending:
            now = self._clock()
            if not self.sched.running and not self._pending:
                nxt = self.sched.next_arrival()
                if realtime and nxt is not None and nxt > now:
                    time.sleep(min(nxt - now, 0.05))
                    continue
            produced = self.step(now)
            if produced == 0 and not self.sched.running and not self._pending and self.sched.waiting:
                head = self.sched.waiting[0]
                if not realtime or head.arrival <= now:
                    # nothing runs, so every page is free, and the oldest arrived request still was not admitted
                    raise RuntimeError(f"request {head.rid} does not fit in the KV cache")
        if self.cuda:
            torch.cuda.synchronize()
        wall = time.perf_counter() - self._t0
        return self.summarise(requests, wall)

    def summarise(self, requests: list[Request], wall: float) -> dict:
        ttft, lat = Percentiles(), Percentiles()
        out_tokens = 0
        for r in requests:
            out_tokens += len(r.output)
            if r.t_first is not None and self._realtime:
                ttft.add(r.t_first - r.arrival)
            if r.t_done is not None and self._realtime:
                lat.add(r.t_done - r.arrival)
        return {"requests": len(requests), "output_tokens": out_tokens, "wall_s": wall,
                "decode_tok_per_s": out_tokens / wall if wall > 0 else float("nan"),
                "prefill_tokens": self.stats["prefill_tokens"], "decode_steps": self.stats["decode_steps"],
                "ttft_p50_s": ttft.pct(50), "ttft_p99_s": ttft.pct(99), "latency_p50_s": lat.pct(50),
                "kv_pages": self.cache.num_pages, "kv_occupancy_end": self.cache.occupancy()}

    def generate(self, prompts: list[list[int]], max_new_tokens: int, eos_token_id: int | None = None,
                 temperature: float = 0.0, top_k: int | None = None) -> list[list[int]]:
        """Offline batched generation through the continuous-batching loop (greedy unless a temperature is given).
        An end-of-sequence token ends a request and is part of its output."""
        self.set_sampling(temperature, top_k)
        reqs = [Request(i, list(p), max_new_tokens, 0.0, eos_token_id) for i, p in enumerate(prompts)]
        self.run(reqs, realtime=False)
        return [r.output for r in reqs]
