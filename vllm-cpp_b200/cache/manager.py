"""The cache manager: paged keys and values with a block table per request, in
groups of layers with the same needs, and slots for per-request state of fixed size.

The reference keeps one pool of blocks for all layers, a ``vector<int32>`` block
table on each Sequence (include/vllm/core/sequence.hpp:54-55) and grows it with
``ensure_sequence_capacity`` with rollback (src/core/block_manager.cpp:82-97);
blocks go back on finish, abort and preemption (src/core/scheduler.cpp:111-121,
168-188).  It has one kind of layer and no per-request state.

Here cache layers whose mixers declare the same PagedKVSpec (kv heads, head size,
window) form a group with pages and tables of its own.  A request holds one table
per group.  A group with a window gives pages back as soon as the window has
passed them: a query at position p reads keys j with p - window < j <= p, so once
a request holds ``n`` tokens no later query reads a key at or below n - window.
A group whose rows stand for ``stride`` tokens each (PagedKVSpec.stride) hands out pages
for n // stride rows; its pool is sized so that whatever fits a group of one row per
token fits it too.  A windowed group that such rows are made from (``keep_block``)
keeps the tokens of the block that is not complete yet, and one whose first tokens stay visible
(``keep_first``) keeps the pages that hold them.
Layers that declare a StateSpec get one slot per live request in a tensor of
their own; the slot is zeroed when the request is admitted.  A request always
gets a slot id, even if no layer has state.

All bookkeeping is host-side and runs without a GPU (``device=None``).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, List, Optional

import numpy as np
import torch

from ..parts.base import CompositeSpec, CompositeView, PagedKVSpec, PagedKVView, StateSpec, StateView, flatten_specs
from .block_pool import BlockPool, PageError

RELEASED = -1     # table entry of a page that a window has passed


class OutOfPages(RuntimeError):
    """A request's next tokens do not fit the free pages of some group."""


@dataclass
class PagedGroup:
    spec: PagedKVSpec
    layers: List[int]                      # cache layer ids, in order
    pool: BlockPool
    pages: Optional[torch.Tensor] = None   # [len(layers), num_pages, planes, kv_heads, page_size * head_dim]: see csrc/common.cuh (kv_pos)


@dataclass
class StateGroup:
    spec: StateSpec
    layers: List[int]
    slots: Optional[torch.Tensor] = None   # [len(layers), num_slots, *shape]


@dataclass
class RequestCache:
    tables: List[List[int]]                # one per paged group
    num_tokens: int = 0
    slot: int = -1
    released: List[int] = field(default_factory=list)   # per group: blocks [0, released) are given back


def cdiv(a: int, b: int) -> int:
    return -(-a // b)


class CacheManager:
    def __init__(self, cache_specs: List[object], page_size: int, num_pages: int, max_num_seqs: int,
                 dtype: torch.dtype = torch.float32, device=None):
        if page_size <= 0:
            raise ValueError("KV block size must be greater than zero")
        self.page_size, self.num_pages, self.max_num_seqs = page_size, num_pages, max_num_seqs
        self.dtype, self.device = dtype, device
        self.paged: List[PagedGroup] = []
        self.state: List[StateGroup] = []
        self._where: List[Optional[tuple]] = []          # cache layer -> ("paged"|"state", group, index in group)
        for layer, spec in enumerate(cache_specs):
            self._where.append(self._register(layer, spec))
        self._free_slots: List[int] = list(range(max_num_seqs - 1, -1, -1))
        self.requests: Dict[object, RequestCache] = {}
        # every group's block tables as rows of one array (see table_rows); widened on demand
        self._table_rows: List[np.ndarray] = [np.full((max_num_seqs, 0), RELEASED, dtype=np.int32) for _ in self.paged]
        if device is not None:
            self._allocate_device()

    def _register(self, layer: int, spec):
        """Where the cache need ``spec`` of cache layer ``layer`` lives: None, ("paged" | "state", group, index in
        group), or ("multi", [one of these per member]) for the mixers of a CompositeSpec."""
        if spec is None:
            return None
        if isinstance(spec, CompositeSpec):
            return ("multi", [self._register(layer, part) for part in spec.parts])
        if isinstance(spec, PagedKVSpec):
            g = next((i for i, pg in enumerate(self.paged) if pg.spec == spec), None)
            if g is None:
                self.paged.append(PagedGroup(spec, [], BlockPool(self.group_pages(spec, self.num_pages, self.max_num_seqs))))
                g = len(self.paged) - 1
            self.paged[g].layers.append(layer)
            return ("paged", g, len(self.paged[g].layers) - 1)
        if isinstance(spec, StateSpec):
            g = next((i for i, sg in enumerate(self.state) if sg.spec == spec), None)
            if g is None:
                self.state.append(StateGroup(spec, []))
                g = len(self.state) - 1
            self.state[g].layers.append(layer)
            return ("state", g, len(self.state[g].layers) - 1)
        raise TypeError(f"cache layer {layer}: unknown cache need {spec!r}")

    @staticmethod
    def group_pages(spec: PagedKVSpec, num_pages: int, max_num_seqs: int) -> int:
        """Pages of the group's pool in a cache of ``num_pages`` pages of one row per token.  With a stride s, requests of
        n_1, n_2, ... tokens that fit those pages hold at most sum(n_i) / s rows, and every request may leave one page
        partly filled: ceil(num_pages / s) + max_num_seqs pages hold them in any mixture."""
        return num_pages if spec.stride == 1 else cdiv(num_pages, spec.stride) + max_num_seqs

    # ---------------------------------------------------------------- device
    @staticmethod
    def bytes_per_page(cache_specs: List[object], page_size: int, dtype: torch.dtype) -> int:
        """Device bytes that one page of tokens costs over all paged cache layers (a group of one row per ``stride``
        tokens costs a page's stride-th part; ``fixed_bytes`` has the rest)."""
        el = torch.empty((), dtype=dtype).element_size()
        return sum(cdiv(s.planes * s.num_kv_heads * page_size * s.head_dim * el, s.stride)
                   for s in flatten_specs(cache_specs) if isinstance(s, PagedKVSpec))

    @staticmethod
    def fixed_bytes(cache_specs: List[object], page_size: int, max_num_seqs: int, dtype: torch.dtype) -> int:
        """Device bytes of the pages that strided groups have beyond their share of the page count (group_pages)."""
        el = torch.empty((), dtype=dtype).element_size()
        return sum((max_num_seqs + 1) * s.planes * s.num_kv_heads * page_size * s.head_dim * el
                   for s in flatten_specs(cache_specs) if isinstance(s, PagedKVSpec) and s.stride > 1)

    def _allocate_device(self) -> None:
        for g in self.paged:
            s = g.spec
            g.pages = torch.zeros((len(g.layers), g.pool.num_blocks, s.planes, s.num_kv_heads, self.page_size * s.head_dim),
                                  dtype=self.dtype, device=self.device)
        for g in self.state:
            g.slots = torch.zeros((len(g.layers), self.max_num_seqs) + tuple(g.spec.shape),
                                  dtype=g.spec.dtype, device=self.device)

    def views(self) -> List[object]:
        """What each cache layer's mixer is handed."""
        return [self._view(w) for w in self._where]

    def _view(self, w):
        if w is None:
            return None
        if w[0] == "multi":
            return CompositeView([self._view(x) for x in w[1]])
        if w[0] == "paged":
            g = self.paged[w[1]]
            return PagedKVView(g.pages[w[2]] if g.pages is not None else None, w[1], self.page_size)
        g = self.state[w[1]]
        return StateView(g.slots[w[2]] if g.slots is not None else None)

    # ------------------------------------------------------------- requests
    def has_free_slot(self) -> bool:
        return bool(self._free_slots)

    def add_request(self, req_id) -> RequestCache:
        if req_id in self.requests:
            raise KeyError(f"request {req_id!r} is already live")
        if not self._free_slots:
            raise OutOfPages(f"all {self.max_num_seqs} request slots are taken")
        slot = self._free_slots.pop()
        rc = RequestCache(tables=[[] for _ in self.paged], slot=slot, released=[0] * len(self.paged))
        self.requests[req_id] = rc
        for t in self._table_rows:
            t[slot, :] = RELEASED
        for g in self.state:
            if g.slots is not None:
                g.slots[:, slot].zero_()
        return rc

    def pages_needed(self, req_id, n_new: int) -> List[int]:
        """Pages each group must still hand out before ``n_new`` more tokens fit."""
        rc = self.requests[req_id]
        n = rc.num_tokens + n_new
        return [max(0, cdiv(n // g.spec.stride, self.page_size) - len(t)) for g, t in zip(self.paged, rc.tables)]

    def _room(self, g: PagedGroup, pages: int) -> int:
        """Most tokens a request may hold with ``pages`` pages of the group."""
        return (pages * self.page_size + 1) * g.spec.stride - 1

    def can_append(self, req_id, n_new: int) -> bool:
        return all(g.pool.can_allocate(n) for g, n in zip(self.paged, self.pages_needed(req_id, n_new)))

    def max_appendable(self, req_id=None) -> int:
        """Most tokens that the request (or, with None, a new request) could take now."""
        if not self.paged:
            return 1 << 30
        if req_id is None:
            return min(self._room(g, g.pool.num_free) for g in self.paged)
        rc = self.requests[req_id]
        return min(self._room(g, len(t) + g.pool.num_free) for g, t in zip(self.paged, rc.tables)) - rc.num_tokens

    def reserve(self, req_id, n_new: int) -> None:
        """Give the request pages for its next ``n_new`` tokens in every group, or none at all."""
        rc = self.requests[req_id]
        need = self.pages_needed(req_id, n_new)
        for g, n in zip(self.paged, need):
            if not g.pool.can_allocate(n):
                raise OutOfPages(f"request {req_id!r} needs {n} more pages for {n_new} tokens; "
                                 f"{g.pool.num_free} of {g.pool.num_blocks} are free")
        for gi, (g, table, n) in enumerate(zip(self.paged, rc.tables, need)):
            for _ in range(n):
                page = g.pool.acquire()
                if len(table) < self._table_rows[gi].shape[1]:
                    self._table_rows[gi][rc.slot, len(table)] = page
                table.append(page)

    def commit(self, req_id, n_new: int) -> None:
        """The request now holds ``n_new`` more tokens; give back what windows have passed."""
        rc = self.requests[req_id]
        rc.num_tokens += n_new
        if any(rc.num_tokens > self._room(g, len(t)) for g, t in zip(self.paged, rc.tables)):
            raise PageError(f"request {req_id!r} holds {rc.num_tokens} tokens but pages for fewer")
        for gi, g in enumerate(self.paged):
            w = g.spec.window
            if w <= 0:
                continue
            # keys at positions <= num_tokens - w are never read again, unless a block's summary is still to be made of them
            dead = rc.num_tokens - w + 1
            if g.spec.keep_block > 1:
                dead = min(dead, rc.num_tokens // g.spec.keep_block * g.spec.keep_block)
            dead_blocks = max(0, dead // self.page_size)
            table = rc.tables[gi]
            # the pages of the first tokens stay
            rc.released[gi] = max(rc.released[gi], cdiv(g.spec.keep_first, self.page_size))
            for b in range(rc.released[gi], min(dead_blocks, len(table))):
                g.pool.release(table[b])
                table[b] = RELEASED
                if b < self._table_rows[gi].shape[1]:
                    self._table_rows[gi][rc.slot, b] = RELEASED
            rc.released[gi] = max(rc.released[gi], min(dead_blocks, len(table)))

    def free_request(self, req_id) -> None:
        rc = self.requests.pop(req_id)
        for g, table in zip(self.paged, rc.tables):
            for b in reversed(table):
                if b != RELEASED:
                    g.pool.release(b)
        self._free_slots.append(rc.slot)

    # ---------------------------------------------------------------- queries
    def num_tokens(self, req_id) -> int:
        return self.requests[req_id].num_tokens

    def table(self, req_id, group: int) -> List[int]:
        return self.requests[req_id].tables[group]

    def table_rows(self, group: int, width: int) -> np.ndarray:
        """The block tables of the group as one int32 array [request slot, width], kept up to date
        with every page handed out or given back (RELEASED where a request holds no page): the
        step function copies rows of it instead of building tables from lists."""
        rows = self._table_rows[group]
        if rows.shape[1] < width:
            wider = np.full((self.max_num_seqs, width), RELEASED, dtype=np.int32)
            for rc in self.requests.values():
                t = rc.tables[group][:width]
                wider[rc.slot, : len(t)] = t
            self._table_rows[group] = rows = wider
        return rows

    def slot(self, req_id) -> int:
        return self.requests[req_id].slot

    def num_free_pages(self) -> int:
        """Free pages of the scarcest group of one row per token (a group with a stride counts rows of another kind)."""
        return min((g.pool.num_free for g in self.paged if g.spec.stride == 1), default=self.num_pages)
