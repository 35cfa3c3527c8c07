"""The cache manager: pages of keys and values with a block table per request, and slots of
fixed-size state per request.

Policy only: this file decides which page holds which positions and when a page goes back; it
launches nothing (the reference keeps the same split, src/block_pool.h:14-15).  Device tensors
are made by ``make_storage`` and handed to the parts as views.

Groups.  Every cache entry of the run order states a need (``PagedKVNeed`` / ``StateNeed`` / none).
Paged entries with the same (kv heads, key and value size, window, chunk) form a *group*: the group has one page
pool and one block table per request, and a page id addresses the same page in every entry of the
group (the reference has one implicit group: one block id spans all layers,
kernels/batch_gpu.cu:75,114-118).  Groups with a window give pages back as soon as every later
query is past them; their block tables then hold -1 at that place.  Groups with chunks (a query reads keys of its own
chunk of positions only) give back the pages of the chunks that have passed.  A need with ``keep_first`` keeps the pages
that hold the positions below it: every later query still reads those.

An entry may also state a ``CompositeNeed``: several needs by name (pages AND a fixed-size state for one mixer;
the needs of mixers that run side by side). Its leaves are placed as above, under the key (cache index, name, ...),
and the entry's view is a dict of the same shape.

Life of a request: ``admit`` (takes a state slot, zeroes its state) -> repeated ``reserve(n)``
(pages for the next n positions in every group, all or nothing) + ``advance(n)`` (the positions
are now filled; pages behind a window are freed) -> ``release`` (everything goes back).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Mapping, Optional, Sequence, Tuple

import torch

from ..parts.base import CompositeNeed, PagedKVNeed, StateNeed


class CacheError(RuntimeError):
    """A misuse of the manager: unknown request, double free, advancing past what was reserved."""


class PagePool:
    """Page ids 0..n-1 with a reference count each. Pages that came back last go out first, so a
    freed page is reused as early as possible."""

    def __init__(self, n_pages: int):
        if n_pages <= 0:
            raise ValueError("a page pool needs at least one page")
        self.n_pages = n_pages
        self._free: List[int] = list(range(n_pages - 1, -1, -1))   # pop() hands out 0 first
        self._ref = [0] * n_pages
        self.peak_in_use = 0

    @property
    def n_free(self) -> int:
        return len(self._free)

    @property
    def n_in_use(self) -> int:
        return self.n_pages - len(self._free)

    def alloc(self) -> Optional[int]:
        if not self._free:
            return None
        p = self._free.pop()
        if self._ref[p] != 0:
            raise CacheError(f"page {p} was on the free list while still referenced")
        self._ref[p] = 1
        self.peak_in_use = max(self.peak_in_use, self.n_in_use)
        return p

    def retain(self, page: int) -> None:
        if self._ref[page] <= 0:
            raise CacheError(f"page {page} is not allocated")
        self._ref[page] += 1

    def free(self, page: int) -> None:
        if not 0 <= page < self.n_pages or self._ref[page] <= 0:
            raise CacheError(f"page {page} freed twice or never allocated")
        self._ref[page] -= 1
        if self._ref[page] == 0:
            self._free.append(page)

    def refcount(self, page: int) -> int:
        return self._ref[page]


@dataclass
class CacheGroup:
    index: int
    need: PagedKVNeed
    cache_ids: List[int]                 # entries of the run order's caches that live in this group
    pool: PagePool
    page_size: int
    k: Optional[torch.Tensor] = None     # [len(cache_ids), n_pages, kv_heads, page_size, head_dim]
    v: Optional[torch.Tensor] = None     # the same with the need's value size last (None: values lie in the key rows)

    @property
    def window(self) -> Optional[int]:
        return self.need.window


@dataclass
class RequestCache:
    rid: Hashable
    slot: int
    length: int = 0                                  # positions filled
    reserved: int = 0                                # positions that have pages (>= length)
    tables: List[List[int]] = field(default_factory=list)   # per group: page id per page index, -1 = given back


@dataclass
class PagedKVView:
    """What an attention part gets for one cache entry."""
    group: int
    k: torch.Tensor          # [n_pages, kv_heads, page_size, head_dim]
    v: Optional[torch.Tensor]  # None where the values are the first channels of the key rows
    page_size: int
    window: Optional[int]


class CacheManager:
    def __init__(self, needs: Mapping[int, object], n_pages: int, page_size: int = 16, n_slots: int = 8):
        """needs: cache index -> PagedKVNeed | StateNeed | None. n_pages: pages in every group's pool."""
        if page_size <= 0:
            raise ValueError("page_size must be positive")
        self.page_size, self.n_slots = page_size, n_slots
        self.groups: List[CacheGroup] = []
        self.group_of_cache: Dict[int, Tuple[int, int]] = {}     # cache id -> (group index, index in group)
        self.state_needs: Dict[int, StateNeed] = {}
        self.state: Dict[int, Dict[str, torch.Tensor]] = {}
        self.needs = dict(needs)
        by_key: Dict[Tuple, CacheGroup] = {}

        def place(key, need):
            """key: the cache index, or (cache index, name, ...) for a leaf of a composite need."""
            if isinstance(need, PagedKVNeed):
                gkey = (need.num_kv_heads, need.head_dim, need.value_dim, need.window, need.values_in_keys,
                        need.keep_first if need.window is not None else 0, need.chunk)
                g = by_key.get(gkey)
                if g is None:
                    g = CacheGroup(len(self.groups), need, [], PagePool(n_pages), page_size)
                    by_key[gkey] = g
                    self.groups.append(g)
                self.group_of_cache[key] = (g.index, len(g.cache_ids))
                g.cache_ids.append(key)
            elif isinstance(need, StateNeed):
                self.state_needs[key] = need
            elif isinstance(need, CompositeNeed):
                for name, sub in need.parts.items():
                    place((key if isinstance(key, tuple) else (key,)) + (name,), sub)
            elif need is not None:
                raise TypeError(f"cache {key}: unknown kind of need {need!r}")

        for cid in sorted(needs):
            place(cid, needs[cid])
        self._free_slots = list(range(n_slots - 1, -1, -1))
        self.requests: Dict[Hashable, RequestCache] = {}

    # ------------------------------------------------------------------ storage

    def make_storage(self, dtype: torch.dtype, device) -> None:
        """Allocates the page tensors of every group and the state tensors of every state entry."""
        for g in self.groups:
            shape = (len(g.cache_ids), g.pool.n_pages, g.need.num_kv_heads, self.page_size)
            g.k = torch.zeros(shape + (g.need.head_dim,), dtype=dtype, device=device)
            g.v = None if g.need.values_in_keys else torch.zeros(shape + (g.need.value_dim,), dtype=dtype, device=device)
        for cid, need in self.state_needs.items():
            # a state tensor declared with dtype None takes the storage's (the compute dtype of the model)
            self.state[cid] = {name: torch.zeros((self.n_slots,) + tuple(shape), dtype=dt or dtype, device=device)
                               for name, (shape, dt) in need.shapes.items()}

    def storage_bytes(self, dtype: torch.dtype) -> int:
        item = torch.empty((), dtype=dtype).element_size()
        return sum(len(g.cache_ids) * g.pool.n_pages * g.need.num_kv_heads * self.page_size *
                   (g.need.head_dim + g.need.stored_value_dim) * item for g in self.groups)

    def view(self, cache_id: int):
        """PagedKVView, the dict of state tensors, a dict of such views by name for a composite need, or None."""
        return self._view(cache_id, self.needs.get(cache_id))

    def _view(self, key, need):
        if isinstance(need, CompositeNeed):
            base = key if isinstance(key, tuple) else (key,)
            return {name: self._view(base + (name,), sub) for name, sub in need.parts.items()}
        if key in self.group_of_cache:
            gi, li = self.group_of_cache[key]
            g = self.groups[gi]
            if g.k is None:
                raise CacheError("make_storage() has not been called")
            return PagedKVView(gi, g.k[li], g.v[li] if g.v is not None else None, self.page_size, g.window)
        if key in self.state_needs:
            return self.state[key]
        return None

    # ------------------------------------------------------------------ requests

    def _req(self, rid) -> RequestCache:
        try:
            return self.requests[rid]
        except KeyError:
            raise CacheError(f"request {rid!r} is not admitted") from None

    def has_slot(self) -> bool:
        return bool(self._free_slots)

    def admit(self, rid) -> RequestCache:
        if rid in self.requests:
            raise CacheError(f"request {rid!r} is already admitted")
        if not self._free_slots:
            raise CacheError("no free request slot")
        slot = self._free_slots.pop()
        for tensors in self.state.values():
            for t in tensors.values():
                t[slot].zero_()
        rc = RequestCache(rid, slot, tables=[[] for _ in self.groups])
        self.requests[rid] = rc
        return rc

    def _first_needed_page(self, g: CacheGroup, length: int) -> int:
        """Index of the first page that a query at position >= length can still read."""
        first = 0 if g.window is None else max(0, length - g.window + 1)
        if g.need.chunk is not None:
            first = max(first, length // g.need.chunk * g.need.chunk)
        return first // self.page_size

    def pages_needed(self, rid, n_new: int) -> List[int]:
        """Per group: pages that reserve(rid, n_new) would take from the pool."""
        rc = self._req(rid)
        end = max(rc.reserved, rc.length + n_new)
        last_page = (end - 1) // self.page_size if end > 0 else -1
        return [max(0, last_page + 1 - len(t)) for t in rc.tables]

    def can_reserve(self, wanted: Sequence[Tuple[Hashable, int]]) -> bool:
        """True if reserve() would succeed for every (rid, n) of the list, taken together."""
        total = [0] * len(self.groups)
        for rid, n in wanted:
            for gi, k in enumerate(self.pages_needed(rid, n)):
                total[gi] += k
        return all(total[gi] <= g.pool.n_free for gi, g in enumerate(self.groups))

    def reserve(self, rid, n_new: int) -> bool:
        """Pages for positions [length, length+n_new) in every group. All or nothing."""
        rc = self._req(rid)
        if n_new < 0:
            raise CacheError("cannot reserve a negative number of positions")
        need = self.pages_needed(rid, n_new)
        if any(k > g.pool.n_free for k, g in zip(need, self.groups)):
            return False
        for g, k, table in zip(self.groups, need, rc.tables):
            for _ in range(k):
                table.append(g.pool.alloc())
        rc.reserved = max(rc.reserved, rc.length + n_new)
        return True

    def unreserve(self, rid) -> None:
        """Gives back pages that were reserved beyond the filled length (a step that did not run)."""
        rc = self._req(rid)
        keep = (rc.length + self.page_size - 1) // self.page_size
        for g, table in zip(self.groups, rc.tables):
            while len(table) > keep:
                p = table.pop()
                if p >= 0:
                    g.pool.free(p)
        rc.reserved = rc.length

    def advance(self, rid, n: int) -> None:
        """The next n positions are filled. Pages that no later query can read go back."""
        rc = self._req(rid)
        if n < 0 or rc.length + n > rc.reserved:
            raise CacheError(f"request {rid!r}: advancing {n} from {rc.length} passes the reserved {rc.reserved}")
        rc.length += n
        for g, table in zip(self.groups, rc.tables):
            first = min(self._first_needed_page(g, rc.length), len(table))
            kept = -(-g.need.keep_first // self.page_size) if g.need.keep_first > 0 else 0      # pages of the kept first positions
            for i in range(kept, first):
                if table[i] >= 0:
                    g.pool.free(table[i])
                    table[i] = -1

    def release(self, rid) -> None:
        rc = self._req(rid)
        for g, table in zip(self.groups, rc.tables):
            for p in table:
                if p >= 0:
                    g.pool.free(p)
            table.clear()
        self._free_slots.append(rc.slot)
        del self.requests[rid]

    # ------------------------------------------------------------------ inspection

    def length(self, rid) -> int:
        return self._req(rid).length

    def slot(self, rid) -> int:
        return self._req(rid).slot

    def block_table(self, rid, group: int) -> List[int]:
        return self._req(rid).tables[group]

    def pages_in_use(self) -> List[int]:
        return [g.pool.n_in_use for g in self.groups]

    def pages_total(self) -> List[int]:
        return [g.pool.n_pages for g in self.groups]

    def pages_free(self) -> List[int]:
        return [g.pool.n_free for g in self.groups]

    def check_invariants(self) -> None:
        """No page lost, held twice, or free while held. For tests."""
        for gi, g in enumerate(self.groups):
            held: Dict[int, int] = {}
            for rc in self.requests.values():
                for p in rc.tables[gi]:
                    if p >= 0:
                        held[p] = held.get(p, 0) + 1
            free = list(g.pool._free)
            if len(set(free)) != len(free):
                raise CacheError(f"group {gi}: a page is on the free list twice")
            for p, n in held.items():
                if n != g.pool.refcount(p):
                    raise CacheError(f"group {gi}: page {p} is held {n} times but counted {g.pool.refcount(p)}")
                if p in free:
                    raise CacheError(f"group {gi}: page {p} is held and free")
            if len(held) + len(free) != g.pool.n_pages:
                raise CacheError(f"group {gi}: {g.pool.n_pages - len(held) - len(free)} pages are lost")
        slots = [rc.slot for rc in self.requests.values()]
        if len(set(slots)) != len(slots) or set(slots) & set(self._free_slots):
            raise CacheError("a state slot is held twice")
        if len(slots) + len(self._free_slots) != self.n_slots:
            raise CacheError("a state slot is lost")
