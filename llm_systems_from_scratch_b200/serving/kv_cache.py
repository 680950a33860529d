"""Cache manager of the serving engine: fixed-size pages (16 tokens by default), a free-list allocator and per-request
block tables.  The reference keeps no KV cache (its ``generate`` recomputes the whole context for
every token, llm-core/llm_core/model.py:210-233); everything here is new capability.

Memory: one K and one V tensor of shape (layers, num_pages, page_size, d_model) in bf16.  For the
1.3B model a page costs 2 * 24 * 16 * 2048 * 2 B = 3 MiB over all layers, so a 180 GB GPU holds tens
of thousands of pages next to the 2.8 GB of weights.

``LayerCache`` is the same for models whose layers differ: every layer run says what it keeps per token
(``PagedSpec``: one vector in a paged pool) or per request (``StateSpec``: a recurrent state in a slot), that it
reads what an earlier run keeps (``SharedSpec``), or several of these (``Parts``).  What a model keeps besides its layers follows
behind them.  All paged layers share the page ids of a request, all recurrent
layers its slot.
"""
from __future__ import annotations

from dataclasses import dataclass

import torch


@dataclass(frozen=True)
class PagedSpec:
    """A layer run that caches ``width`` activations per token."""
    width: int


@dataclass(frozen=True)
class StateSpec:
    """A state of this shape per request: "float32", in the type of the activations ("activations") or a number of tokens ("tokens")."""
    shape: tuple
    kind: str = "float32"


@dataclass(frozen=True)
class SharedSpec:
    """A layer run that keeps nothing of its own and reads the entry of an earlier run."""
    run: int


@dataclass(frozen=True)
class Parts:
    """A layer run that keeps several things; its entry is a tuple."""
    specs: tuple


def flatten(specs) -> list:
    out = []
    for s in specs:
        out += flatten(s.specs) if isinstance(s, Parts) else [s]
    return out


class PageAllocator:
    """LIFO free list over page ids.  The list lives in the C++ host runtime when that library is available
    (``utils.host_runtime``), otherwise in a Python list; both hand pages out in the same order."""

    def __init__(self, num_pages: int, native: bool | None = None):
        self.num_pages = num_pages
        self._pool = None
        if native is not False:
            try:
                from ..utils import host_runtime
                if host_runtime.available():
                    self._pool = host_runtime.NativePagePool(num_pages)
            except Exception:
                self._pool = None
        if native is True and self._pool is None:
            raise RuntimeError("host runtime library is not available")
        self._free = list(range(num_pages - 1, -1, -1)) if self._pool is None else None

    @property
    def free(self) -> int:
        return self._pool.free if self._pool is not None else len(self._free)

    def take(self, n: int) -> list[int]:
        if self._pool is not None:
            return self._pool.take(n)
        if n > len(self._free):
            raise MemoryError(f"out of KV pages: want {n}, have {len(self._free)}")
        out = self._free[-n:][::-1] if n else []
        del self._free[len(self._free) - n:]
        return out

    def give(self, pages: list[int]):
        if self._pool is not None:
            return self._pool.give(pages)
        self._free.extend(reversed(pages))


class PagedKVCache:
    def __init__(self, n_layers: int, d_model: int, num_pages: int, page_size: int = 16, device="cuda",
                 dtype=torch.bfloat16):
        self.n_layers, self.d_model, self.page_size, self.num_pages = n_layers, d_model, page_size, num_pages
        self.k = torch.zeros((n_layers, num_pages, page_size, d_model), dtype=dtype, device=device)
        self.v = torch.zeros((n_layers, num_pages, page_size, d_model), dtype=dtype, device=device)
        self.allocator = PageAllocator(num_pages)
        self.slot_allocator = None                 # nothing is carried per request besides its pages

    @staticmethod
    def pages_for(tokens: int, page_size: int = 16) -> int:
        return -(-tokens // page_size)

    @staticmethod
    def bytes_per_page(n_layers: int, d_model: int, page_size: int = 16, itemsize: int = 2) -> int:
        return 2 * n_layers * page_size * d_model * itemsize

    def occupancy(self) -> float:
        return 1.0 - self.allocator.free / max(1, self.num_pages)

    def slots(self, pages: list[int], start: int, count: int) -> list[int]:
        """Flat cache slots (page * page_size + offset) of token positions [start, start + count)."""
        ps = self.page_size
        if self.allocator._pool is not None and count > 64:
            from ..utils import host_runtime
            return host_runtime.slots(pages, ps, start, count)
        return [pages[t // ps] * ps + t % ps for t in range(start, start + count)]


class LayerCache:
    """Paged pools and state slots, one entry per layer run in ``entries``.

    Freed pages and slots are handed out again as they are: a position's cached vector is written before anything reads
    it, and a recurrent layer starts from the zero state at position 0 whatever the slot held."""

    def __init__(self, specs: list, num_pages: int, page_size: int, num_slots: int, device, dtype):
        self.specs, self.page_size, self.num_pages, self.num_slots = specs, page_size, num_pages, num_slots
        self.entries = []
        types = {"float32": torch.float32, "activations": dtype, "tokens": torch.int32}

        def entry(s):
            if isinstance(s, Parts):
                return tuple(entry(p) for p in s.specs)
            if isinstance(s, PagedSpec):
                return torch.zeros((num_pages, page_size, s.width), dtype=dtype, device=device)
            if isinstance(s, StateSpec):
                return torch.zeros((num_slots, *s.shape), dtype=types[s.kind], device=device)
            return self.entries[s.run] if isinstance(s, SharedSpec) else None
        for s in specs:
            self.entries.append(entry(s))
        self.allocator = PageAllocator(num_pages)
        self.slot_allocator = PageAllocator(num_slots)

    @staticmethod
    def bytes_per_page(specs: list, page_size: int, itemsize: int) -> int:
        return sum(s.width for s in flatten(specs) if isinstance(s, PagedSpec)) * page_size * itemsize

    @staticmethod
    def bytes_per_slot(specs: list, itemsize: int = 4) -> int:
        total = 0
        for s in flatten(specs):
            if isinstance(s, StateSpec):
                n = itemsize if s.kind == "activations" else 4
                for k in s.shape:
                    n *= k
                total += n
        return total

    def occupancy(self) -> float:
        return 1.0 - self.allocator.free / max(1, self.num_pages)
