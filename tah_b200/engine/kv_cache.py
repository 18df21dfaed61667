"""Paged KV cache with one page pool and one page table per iteration depth.

The reference grows a dense ``(B, n, heads, hd)`` tensor per ``(layer, depth)`` slot with
``torch.cat`` on every step (reference ``tah/model/causal_cache.py:84-95``) and pads the
depth->=1 slots over the whole batch.  Here each depth has a pool of fixed-size pages

    pool[depth]: [layers, pages, 2 (K,V), kv_heads, page_size, head_dim]   bf16

and a row owns only the pages its real entries need; the depth->=1 pools hold hard-token
entries only.  Free pages are handed out on the device (``free_stack``/``free_count``,
popped by the tick kernel), so decode never returns to the host for memory.

A model whose layers differ gives ``CacheGeometry.layers``: one :class:`LayerKV` per layer with its own K and V sizes, or
``None`` for a layer without keys (a recurrent layer), or ``LayerKV(shared_with=j)`` for a layer that reads the cache of
layer ``j``.  All layers share one page table; the pool of a layer is then a tensor of its own with the same page layout
``[K: kv_heads, page_size, k_dim][V: kv_heads, page_size, v_dim]``.  Beside it a layer may have further pools under the same page
table: ``factors``, one fp32 number per token, and ``pooled``, the means of blocks of ``block`` keys.  A page holds
``pool_rows`` of those (a power of two, at least ``page_size / block``), so block ``b`` is row ``b % pool_rows`` of the row's
logical page ``b // pool_rows``, which the row owns by the time the block is complete.  What recurrent layers carry from token to token
lives beside the pages in :class:`RecurrentState`, one slot per cache row.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence, Tuple

import os

import torch


@dataclass
class LayerKV:
    kv_heads: int = 0
    k_dim: int = 0
    v_dim: int = 0
    shared_with: Optional[int] = None     # the layer whose pool this layer reads
    factor: bool = False                  # one fp32 number per token beside the keys
    block: Optional[int] = None           # keys of a pooled block; None: no pooled blocks

    def pool_rows(self, page_size: int) -> int:
        """Pooled blocks that a page has room for."""
        n = 1
        while self.block is not None and n * self.block < page_size:
            n *= 2
        return 0 if self.block is None else n


@dataclass
class CacheGeometry:
    n_layers: int
    n_kv_heads: int
    head_dim: int
    page_size: int = 16
    layers: Optional[List[Optional[LayerKV]]] = None

    @classmethod
    def per_layer(cls, layers: Sequence[Optional[LayerKV]], page_size: int = 16) -> "CacheGeometry":
        for i, l in enumerate(layers):
            if l is not None and l.shared_with is not None:
                j = l.shared_with
                if not 0 <= j < len(layers) or layers[j] is None or layers[j].shared_with is not None:
                    raise ValueError(f"layer {i} shares the cache of layer {j}, which has none of its own")
        return cls(len(layers), 0, 0, page_size, list(layers))


GUARD_PATTERN = 0x5A5A          # int16 view of the bf16 guard pages


class PagedKVCache:
    def __init__(self, geo: CacheGeometry, rows: int, max_tokens_per_row: int, n_depths: int,
                 deep_fraction: float = 0.25, device="cuda", dtype=torch.bfloat16, pool_tokens: Optional[int] = None):
        """``pool_tokens``: capacity of the depth-0 pool in tokens, when it is not ``rows * max_tokens_per_row`` (rows
        then compete for pages)."""
        self.geo, self.rows, self.n_depths = geo, rows, n_depths
        self.page_size = geo.page_size
        ppr = (max_tokens_per_row + geo.page_size - 1) // geo.page_size + 1
        self.max_pages = [ppr] * n_depths
        self.n_pages: List[int] = []
        self.pool: List = []              # per depth: one tensor, or with geo.layers a list with one tensor (or None) per layer
        self.factors: List[List[Optional[torch.Tensor]]] = []     # per depth and layer (see the module docstring)
        self.pooled: List[List[Optional[torch.Tensor]]] = []
        self.page_table: List[torch.Tensor] = []
        self.len: List[torch.Tensor] = []
        self.free_stack: List[torch.Tensor] = []
        self.free_count: List[torch.Tensor] = []
        # TAH_B200_CANARY=G: G guard pages behind every layer's pool, filled with a bit pattern that no kernel may
        # touch (pages are only ever handed out from the free stack); check_guards() verifies them on the host
        self.guard_pages = int(os.environ.get("TAH_B200_CANARY", "0") or 0)
        for d in range(n_depths):
            pages = rows * ppr if d == 0 else max(rows * 2, int(rows * ppr * deep_fraction))
            if d == 0 and pool_tokens is not None:
                pages = max(1, (pool_tokens + geo.page_size - 1) // geo.page_size)
            self.n_pages.append(pages)
            if geo.layers is None:
                pool = torch.zeros(geo.n_layers, pages + self.guard_pages, 2, geo.n_kv_heads, geo.page_size, geo.head_dim,
                                   dtype=dtype, device=device)
            else:
                pool = [None if l is None or l.shared_with is not None else
                        torch.zeros(pages + self.guard_pages, l.kv_heads * geo.page_size * (l.k_dim + l.v_dim), dtype=dtype,
                                    device=device) for l in geo.layers]
            self.pool.append(pool)
            self.factors.append([None if l is None or not l.factor else
                                 torch.zeros(pages + self.guard_pages, geo.page_size, device=device) for l in geo.layers or []])
            self.pooled.append([None if l is None or l.block is None else
                                torch.zeros(pages + self.guard_pages, l.kv_heads * l.pool_rows(geo.page_size) * l.k_dim, dtype=dtype,
                                            device=device) for l in geo.layers or []])
            if self.guard_pages:
                for t in self._pools(d):
                    t[..., pages:, :].view(torch.int16).fill_(GUARD_PATTERN)
            self.page_table.append(torch.zeros(rows, ppr, dtype=torch.int32, device=device))
            self.len.append(torch.zeros(rows, dtype=torch.int32, device=device))
            self.free_stack.append(torch.arange(pages, dtype=torch.int32, device=device))
            self.free_count.append(torch.full((1,), pages, dtype=torch.int32, device=device))

    def check_guards(self) -> bool:
        """True when every guard page still holds the pattern (always true without ``TAH_B200_CANARY``)."""
        if not self.guard_pages:
            return True
        return all(bool((t[..., n:, :].view(torch.int16) == GUARD_PATTERN).all())
                   for d, n in enumerate(self.n_pages) for t in self._pools(d))

    def _pools(self, depth: int) -> List[torch.Tensor]:
        """The pool tensors of a depth as ``[..., pages, elements of a page]`` views."""
        p = self.pool[depth]
        if self.geo.layers is None:
            return [p.flatten(2)]
        return [t for t in p + self.factors[depth] + self.pooled[depth] if t is not None]

    def bytes(self) -> int:
        return sum(t.numel() * t.element_size() for d in range(self.n_depths) for t in self._pools(d))

    def reset(self) -> None:
        for d in range(self.n_depths):
            self.len[d].zero_()
            self.page_table[d].zero_()
            self.free_stack[d].copy_(torch.arange(self.n_pages[d], dtype=torch.int32, device=self.free_stack[d].device))
            self.free_count[d].fill_(self.n_pages[d])

    def layer_pool(self, depth: int, layer: int) -> Optional[torch.Tensor]:
        """The pool a layer reads (its own or the one it shares); None for a layer without keys."""
        l = self.geo.layers[layer] if self.geo.layers is not None else None
        if l is not None and l.shared_with is not None:
            layer = l.shared_with
        return self.pool[depth][layer]

    def assign_prefill(self, depth: int, counts: torch.Tensor) -> torch.Tensor:
        """Give each row ``ceil(counts[r] / page_size)`` pages from the top of the free stack, set
        ``len`` and the page table (host-side, once per request batch).  Returns for every one of the
        ``sum(counts)`` entries, in row-major order, its slot ``page * page_size + offset``."""
        ps = self.page_size
        dev = self.len[depth].device
        counts = counts.to(device=dev, dtype=torch.int64)
        need = (counts + ps - 1) // ps
        total = int(need.sum())
        free = int(self.free_count[depth])
        if total > free or int(need.max() if need.numel() else 0) > self.max_pages[depth]:
            raise RuntimeError(f"KV pool of depth {depth} too small: need {total} pages, {free} free")
        first = torch.cumsum(need, 0) - need                     # first page rank of each row
        # pages are taken from the top of the stack: rank k -> stack[free - 1 - k]
        row_of_page = torch.repeat_interleave(torch.arange(self.rows, device=dev), need)
        rank = torch.arange(total, device=dev)
        page_ids = self.free_stack[depth][(free - 1 - rank).long()]
        col = rank - first[row_of_page]
        self.page_table[depth][row_of_page, col] = page_ids
        self.free_count[depth].fill_(free - total)
        self.len[depth].copy_(counts.to(torch.int32))
        # slots of the entries
        row_of_entry = torch.repeat_interleave(torch.arange(self.rows, device=dev), counts)
        start = torch.cumsum(counts, 0) - counts
        j = torch.arange(int(counts.sum()), device=dev) - start[row_of_entry]
        pg = self.page_table[depth][row_of_entry, (j // ps)].long()
        return (pg * ps + j % ps).to(torch.int32)

    def assign_rows(self, depth: int, rows: torch.Tensor, counts: torch.Tensor) -> torch.Tensor:
        """Like :meth:`assign_prefill` for a subset of rows (request admission while other rows keep decoding):
        ``rows [n]`` get ``counts [n]`` entries each; the other rows' lengths and pages are untouched.  The rows
        must be empty at this depth (see :meth:`free_rows`).  Returns the slots of the entries, row-major."""
        ps = self.page_size
        dev = self.len[depth].device
        rows = rows.to(device=dev, dtype=torch.int64)
        counts = counts.to(device=dev, dtype=torch.int64)
        need = (counts + ps - 1) // ps
        total = int(need.sum())
        free = int(self.free_count[depth])
        if total > free or int(need.max() if need.numel() else 0) > self.max_pages[depth]:
            raise RuntimeError(f"KV pool of depth {depth} too small: need {total} pages, {free} free")
        first = torch.cumsum(need, 0) - need
        which = torch.repeat_interleave(torch.arange(rows.numel(), device=dev), need)
        rank = torch.arange(total, device=dev)
        page_ids = self.free_stack[depth][(free - 1 - rank).long()]
        col = rank - first[which]
        self.page_table[depth][rows[which], col] = page_ids
        self.free_count[depth].fill_(free - total)
        self.len[depth][rows] = counts.to(torch.int32)
        which_e = torch.repeat_interleave(torch.arange(rows.numel(), device=dev), counts)
        start = torch.cumsum(counts, 0) - counts
        j = torch.arange(int(counts.sum()), device=dev) - start[which_e]
        pg = self.page_table[depth][rows[which_e], (j // ps)].long()
        return (pg * ps + j % ps).to(torch.int32)

    def free_rows(self, rows: torch.Tensor) -> int:
        """Return every page of ``rows`` (all depths) to the free stacks and clear their lengths.  Call between
        ticks.  Returns the number of pages released."""
        ps = self.page_size
        released = 0
        for d in range(self.n_depths):
            dev = self.len[d].device
            r = rows.to(device=dev, dtype=torch.int64)
            n = (self.len[d][r].to(torch.int64) + ps - 1) // ps
            total = int(n.sum())
            if total:
                which = torch.repeat_interleave(r, n)
                first = torch.cumsum(n, 0) - n
                col = torch.arange(total, device=dev) - torch.repeat_interleave(first, n)
                pages = self.page_table[d][which, col]
                free = int(self.free_count[d])
                self.free_stack[d][free:free + total] = pages
                self.free_count[d].fill_(free + total)
                released += total
            self.len[d][r] = 0
        return released

    def pages_in_use(self, depth: int) -> int:
        return self.n_pages[depth] - int(self.free_count[depth])


class RecurrentState:
    """fp32 state that recurrent layers carry from token to token: for each layer a tuple of tensors whose first
    dimension is the cache row (a row's slot is its row number).  Kernels start a sequence from zeros at position 0, so a
    row that changes hands needs no clearing."""

    def __init__(self, shapes: Sequence[Optional[Sequence[Tuple[int, ...]]]], rows: int, device="cuda"):
        self.rows = rows
        self.layers = [None if sh is None else tuple(torch.zeros(rows, *s, dtype=torch.float32, device=device) for s in sh)
                       for sh in shapes]

    def bytes(self) -> int:
        return sum(t.numel() * 4 for l in self.layers if l is not None for t in l)
