"""One step of the model: which tokens of which requests run, where they are cached, and what the kernels need to know.

A step is one batch of rows.  Rows [0, n_single) are running requests that bring one token each (a decode step; row i is
sequence i); the rows behind them are the portions of prompts, request after request (``cu`` counts from row n_single).  A portion
may start anywhere in its request: its earlier tokens are in the cache and the state."""
from __future__ import annotations

from dataclasses import dataclass, field

import numpy as np
import torch


@dataclass
class StepBatch:
    tokens: torch.Tensor                 # (R,) int64
    positions: torch.Tensor              # (R,) int32, position of the token inside its request
    slots: torch.Tensor                  # (R,) int64 cache slot (page * page_size + offset); negative = padding row
    tables: torch.Tensor                 # (sequences, max_pages) int32 page ids
    ctx: torch.Tensor                    # (n_single,) int32 tokens a single row can see (position + 1)
    state_slots: torch.Tensor            # (sequences,) int32 recurrent state; negative = padding row
    row_seq: torch.Tensor                # (R,) int32 sequence of the row
    n_single: int
    cu: torch.Tensor | None = None       # (portions + 1,) int32
    portions: list = field(default_factory=list)     # (start position, tokens) of every portion
    splits: int = 0                      # context splits of the decode attention (0 = choose)
    order: list = field(default_factory=list)        # entry index of each sequence, as the caller listed them
    gathered: dict = field(default_factory=dict)     # packed cache rows of this pass over the layers, for layers that share a cache
    _ranges: dict = field(default_factory=dict)

    @property
    def n_rows(self) -> int:
        return self.tokens.numel()

    @property
    def max_portion(self) -> int:
        return max((n for _, n in self.portions), default=0)

    @property
    def spans(self) -> list[tuple[int, int]]:
        out, at = [], 0
        for _, n in self.portions:
            out.append((at, at + n))
            at += n
        return out

    def key_ranges(self, window: int):
        """Keys that the portions can see under a sliding window (0 = none): device cu_k (portions + 1,), first position
        per portion, and the host's (total keys, longest range).  Computed once per window and step."""
        got = self._ranges.get(window)
        if got is None:
            first = [max(0, s - window + 1) if window > 0 else 0 for s, _ in self.portions]
            lens = [s + n - f for (s, n), f in zip(self.portions, first)]
            cu = np.zeros(len(lens) + 1, dtype=np.int32)
            cu[1:] = np.cumsum(lens)
            dev = self.tokens.device
            got = self._ranges[window] = (_to(cu, dev), _to(np.asarray(first, dtype=np.int32), dev), int(cu[-1]), max(lens))
        return got

    def chunk_ranges(self, tokens: int):
        """Chunks of ``tokens`` that the portions consist of: device offsets (portions + 1,) and their number.  Computed once per step."""
        got = self._ranges.get(("chunks", tokens))
        if got is None:
            cu = np.zeros(len(self.portions) + 1, dtype=np.int32)
            cu[1:] = np.cumsum([-(-n // tokens) for _, n in self.portions])
            got = self._ranges["chunks", tokens] = (_to(cu, self.tokens.device), int(cu[-1]))
        return got

    @classmethod
    def build(cls, entries, page_size: int, max_pages: int, device) -> "StepBatch":
        """``entries``: (request, start position, token ids); the requests' pages cover the tokens."""
        one = [len(ids) == 1 and start > 0 for _, start, ids in entries]      # a request's first token is a portion
        order = sorted(range(len(entries)), key=lambda i: not one[i])         # stable: single tokens first
        n_single = sum(one)
        tok, pos, slot, seq = [], [], [], []
        tables = np.zeros((len(entries), max_pages), dtype=np.int32)
        state = np.empty(len(entries), dtype=np.int32)
        for k, i in enumerate(order):
            req, start, ids = entries[i]
            p = np.arange(start, start + len(ids), dtype=np.int64)
            pages = np.asarray(req.pages, dtype=np.int64)
            tok.append(np.asarray(ids, dtype=np.int64))
            pos.append(p.astype(np.int32))
            slot.append(pages[p // page_size] * page_size + p % page_size)
            seq.append(np.full(len(ids), k, dtype=np.int32))
            tables[k, :len(pages)] = pages
            state[k] = req.slot
        portions = [(entries[i][1], len(entries[i][2])) for i in order[n_single:]]
        cu = np.zeros(len(portions) + 1, dtype=np.int32)
        cu[1:] = np.cumsum([n for _, n in portions]) if portions else []
        pos = np.concatenate(pos)
        up = lambda a: _to(a, device)
        return cls(up(np.concatenate(tok)), up(pos), up(np.concatenate(slot)), up(tables), up(pos[:n_single] + 1), up(state),
                   up(np.concatenate(seq)), n_single, up(cu) if portions else None, portions, 0, order)

    def last_rows(self) -> np.ndarray:
        """Row of the last token of every entry, in the order the caller listed the entries."""
        return self.rows_of([-1] * len(self.order))

    def rows_of(self, places) -> np.ndarray:
        """Row of token ``places[i]`` (negative: from the end) of entry i."""
        start, length = self._starts()
        out = np.empty(len(self.order), dtype=np.int64)
        for k, i in enumerate(self.order):
            w = places[i]
            out[i] = start[k] + (w if w >= 0 else length[k] + w)
        return out

    def wanted_rows(self, want) -> np.ndarray:
        """Rows of the wanted tokens: ``want[i]`` lists places in entry i; entry by entry."""
        start, length = self._starts()
        at = {i: (start[k], length[k]) for k, i in enumerate(self.order)}
        rows = []
        for i, places in enumerate(want):
            a, n = at[i]
            for w in places:
                if not 0 <= w < n:
                    raise ValueError(f"place {w} is outside the entry's {n} tokens")
                rows.append(a + w)
        return np.asarray(rows, dtype=np.int64)

    def _starts(self):
        length = [1] * self.n_single + [n for _, n in self.portions]
        return [0, *np.cumsum(length)[:-1].tolist()] if length else [], length


def _to(a: np.ndarray, device) -> torch.Tensor:
    t = torch.from_numpy(np.ascontiguousarray(a))
    if torch.device(device).type == "cuda":
        return t.pin_memory().to(device, non_blocking=True)
    return t
