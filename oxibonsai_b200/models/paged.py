"""Page and state bookkeeping shared by the device caches.

Reference: ``BlockPool`` / ``BlockTable`` (crates/oxibonsai-model/src/paged_kv_cache.rs:33-557) for the pages; recurrent state
has no counterpart there.  ``PagePool`` hands out reference-counted pages; the caches (``PagedKvCache`` in ``qwen3``,
``RowCache`` here) own the tensors the pages index.  ``StatePool`` hands out one state row per sequence.
"""
from __future__ import annotations

import torch


class PagePool:
    """Reference-counted pages; ``on_exhausted(missing)`` may free pages when an allocation does not fit."""

    def __init__(self, num_pages: int, page_size: int):
        self.num_pages, self.page_size = num_pages, page_size
        self.free_pages = list(range(num_pages - 1, -1, -1))
        self.refcount = [0] * num_pages        # pages may be shared between sequences and the prefix cache
        self.on_exhausted = None               # optional callback(n_missing) that may free pages (prefix-cache eviction)

    def alloc(self, n: int) -> list[int]:
        if n > len(self.free_pages) and self.on_exhausted is not None:
            self.on_exhausted(n - len(self.free_pages))
        if n > len(self.free_pages):
            raise MemoryError(f"KV cache exhausted: need {n} pages, {len(self.free_pages)} free")
        pages = [self.free_pages.pop() for _ in range(n)]
        for p in pages:
            self.refcount[p] = 1
        return pages

    def retain(self, pages: list[int]) -> None:
        for p in pages:
            self.refcount[p] += 1

    def release(self, pages: list[int]) -> None:
        for p in reversed(pages):
            self.refcount[p] -= 1
            if self.refcount[p] <= 0:
                self.refcount[p] = 0
                self.free_pages.append(p)

    @property
    def utilization(self) -> float:
        return 1.0 - len(self.free_pages) / max(1, self.num_pages)


class RowCache(PagePool):
    """Paged cache of attention layers: per layer ``rows`` [pages, kv_heads, page_size, row] and, by what they hold, a companion:
    "separate": keys, with ``values`` of the same shape; "shared": rows that serve as key and value, with one float per row
    (``factors``: the key's reciprocal root mean square); "latent": rows that keys and values are expanded from, alone.
    ``layers``: {layer index: (kv heads, row elements, kind)}; layers may differ, they share the page numbering."""

    def __init__(self, layers: dict[int, tuple[int, int, str]], num_pages: int, page_size: int, kvt: int, dtype: torch.dtype, device):
        super().__init__(num_pages, page_size)
        self.kvt = kvt
        self.rows, self.values, self.factors = {}, {}, {}
        for l, (h, row, kind) in layers.items():
            new = lambda *shape, dtype=dtype: torch.zeros((num_pages, h, page_size, *shape), dtype=dtype, device=device)
            self.rows[l] = new(row)
            if kind == "separate":
                self.values[l] = new(row)
            elif kind == "shared":
                self.factors[l] = new(dtype=torch.float32)

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * t.element_size() for d in (self.rows, self.values, self.factors) for t in d.values())


class StatePool:
    """Recurrent state of ``num_rows`` sequences: per layer a set of f32 tensors whose first dimension is the state row.
    ``layers``: {layer index: {name: shape of one row}}.  A row is not cleared when it is handed out: a recurrence starts from
    zero at position 0 whatever the row holds."""

    def __init__(self, layers: dict[int, dict[str, tuple[int, ...]]], num_rows: int, device):
        self.num_rows = num_rows
        self.free_rows = list(range(num_rows - 1, -1, -1))
        self.tensors = {l: {k: torch.zeros((num_rows, *shape), dtype=torch.float32, device=device) for k, shape in d.items()}
                        for l, d in layers.items()}

    def alloc(self) -> int:
        if not self.free_rows:
            raise MemoryError(f"recurrent state exhausted: all {self.num_rows} rows are in use")
        return self.free_rows.pop()

    def release(self, row: int) -> None:
        self.free_rows.append(row)

    @property
    def nbytes(self) -> int:
        return sum(t.numel() * 4 for d in self.tensors.values() for t in d.values())
