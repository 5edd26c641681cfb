"""The cache manager: pages of keys and values with a block table per request, and
fixed-size state slots per request.

Calls of the run order that need keys and values of the same shape and reach (all
positions, or a window of them) form a *group*.  A group has its own pool of pages,
its own key and value tensors [calls, pages, page_size, kv_heads, head_dim] and its
own block table per request, so a windowed group can give pages back while a
full-attention group keeps them.  Calls that need a record of fixed size get a
float32 tensor [slots, *shape]; a request holds one slot id for all of them, even in
an architecture that has no such call.  A slot's records are zero when a request
receives it (`add` clears them), so no mixer ever sees its slot's previous holder.

A group may hold one row per `every` tokens instead of one per token (pooled blocks: a row
stands for that many positions).  Its tables and its pool count rows, so both are shorter by that
factor; every live request may begin a page of its own, so the pool has one page per request more.

A request's pages are given back when it ends (`free`) and, in a group whose reach
is bounded (a window, or chunks that do not see one another), as soon as every slot of
the page lies behind what any future query can see (`advance`).  Released block-table entries read -1; no kernel touches them because
the window bound excludes their positions.  Where a window keeps its first positions visible, their
pages stay as long as the request lives.

In the reference the same duties are split between `KvStorage` (per-layer K and V
tensors [num_blocks, block_size, kv_heads, head_dim], src/kv_storage.rs:7, 92-98),
`ConvCache` (hash maps keyed by (sequence, layer), src/conv_cache.rs:33-41) and the
external scheduler crate's block tables (src/engine.rs:375-387).
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional, Sequence

import numpy as np
import torch

from ..errors import CacheError
from ..parts.base import PagedNeed, SeveralNeeds, StateNeed
from .pages import PagePool


@dataclass
class CacheView:
    """What one call of the run order sees of the cache."""
    kind: str                          # "paged", "state" or "several"
    owns: bool                         # False: reads the cache another call writes
    group: int = -1                    # paged: index into StepContext.groups
    k: Optional[torch.Tensor] = None   # paged: [pages, page_size, kv_heads, head_dim]
    v: Optional[torch.Tensor] = None
    state: Optional[torch.Tensor] = None   # state: float32 [slots, *shape]
    parts: Optional[list] = None       # several: one view (or None) per branch of the mixer


@dataclass
class Group:
    need: PagedNeed
    calls: List[int]
    pool: PagePool
    k: Optional[torch.Tensor] = None
    v: Optional[torch.Tensor] = None


class PageTable:
    """A request's page ids in one group, logical page -> physical page (-1 once released).
    Kept in a numpy array so that a step's batch packing copies it without conversion;
    indexing and slicing give Python ints and lists."""

    __slots__ = ("_a", "_n")

    def __init__(self):
        self._a = np.empty(16, dtype=np.int32)
        self._n = 0

    def append(self, page: int) -> None:
        if self._n == self._a.shape[0]:
            grown = np.empty(2 * self._n, dtype=np.int32)
            grown[:self._n] = self._a
            self._a = grown
        self._a[self._n] = page
        self._n += 1

    def view(self, n: Optional[int] = None) -> np.ndarray:
        return self._a[:self._n if n is None else n]

    def __len__(self) -> int:
        return self._n

    def __getitem__(self, i):
        out = self._a[:self._n][i]
        return out.tolist() if isinstance(i, slice) else int(out)

    def __setitem__(self, i: int, page: int) -> None:
        self._a[:self._n][i] = page

    def __iter__(self):
        return iter(self._a[:self._n].tolist())

    def __eq__(self, other):
        return list(self) == list(other)

    def __repr__(self):
        return f"PageTable({list(self)})"


@dataclass
class RequestCache:
    slot: int
    tokens: int = 0                              # positions covered by reserved pages
    computed: int = 0                            # positions whose keys are written
    tables: List[PageTable] = field(default_factory=list)    # per group, -1 = released
    first_live: List[int] = field(default_factory=list)     # per group: first page kept


class CacheManager:
    def __init__(self, needs: Sequence[Optional[object]], cache_of: Sequence[Optional[int]],
                 page_size: int, num_pages: int, max_requests: int,
                 dtype: torch.dtype = torch.float32, device="cpu", allocate: bool = True):
        """needs[i]: PagedNeed, StateNeed, SeveralNeeds (a mixer of several mixers: each part is
        handled as a call of its own, named (i, part)) or None for call i of the run order;
        cache_of[i]: the call whose cache call i reads, or None.  `num_pages` pages per
        group; `max_requests` state slots.  `allocate=False` keeps only the
        bookkeeping (for tests and planning)."""
        if page_size < 1:
            raise CacheError(f"page size must be at least 1, got {page_size}")
        self.page_size = page_size
        self.num_pages = num_pages
        self.max_requests = max_requests
        self.dtype = dtype
        self.device = device
        self.groups: List[Group] = []
        self.states: Dict[int, torch.Tensor] = {}
        self.slots = PagePool(max_requests, "state slot")
        self.requests: Dict[Hashable, RequestCache] = {}
        self._views: List[Optional[CacheView]] = [None] * len(needs)
        call_group: Dict[int, int] = {}
        state_calls: Dict[tuple, List[int]] = {}
        def flatten(name, need):
            """(name, need) of every part, however deep: part j of `name` is (name, j)."""
            if not isinstance(need, SeveralNeeds):
                return [(name, need)]
            return [x for j, part in enumerate(need.parts) for x in flatten((name, j), part)]

        flat = []
        for i, need in enumerate(needs):
            if isinstance(need, SeveralNeeds) and cache_of[i] is not None:
                raise CacheError(f"call {i}: a mixer of several mixers keeps its own caches")
            flat += flatten(i, need)
        for i, need in flat:
            if isinstance(need, PagedNeed):
                gi = next((g for g, grp in enumerate(self.groups) if grp.need == need), None)
                if gi is None:
                    gi = len(self.groups)
                    pages = num_pages if need.every == 1 else \
                        -(-num_pages // need.every) + max_requests
                    self.groups.append(Group(need, [], PagePool(pages)))
                self.groups[gi].calls.append(i)
                call_group[i] = gi
            elif isinstance(need, StateNeed):
                state_calls.setdefault(tuple(need.shape), []).append(i)
                self.states[i] = None
            elif need is not None:
                raise CacheError(f"call {i}: unknown cache need {need!r}")
        # calls whose records have the same shape share one tensor [calls, slots, *shape],
        # so that a slot is cleared for all of them at once
        self._state_blocks: List[torch.Tensor] = []
        if allocate:
            for shape, calls in state_calls.items():
                block = torch.zeros((len(calls), max_requests) + shape, dtype=torch.float32,
                                    device=device)
                self._state_blocks.append(block)
                for ci, i in enumerate(calls):
                    self.states[i] = block[ci]
        for grp in self.groups:
            if allocate:
                shape = (len(grp.calls), grp.pool.num_pages, page_size, grp.need.num_kv_heads)
                grp.k = torch.zeros(shape + (grp.need.head_dim,), dtype=dtype, device=device)
                grp.v = torch.zeros(shape + (grp.need.value_dim,), dtype=dtype, device=device)
        def view(src, owns):
            if src in call_group:
                grp = self.groups[call_group[src]]
                ci = grp.calls.index(src)
                return CacheView("paged", owns, call_group[src], grp.k[ci] if allocate else None,
                                 grp.v[ci] if allocate else None)
            if src in self.states:
                return CacheView("state", owns, state=self.states[src])
            return None

        def several(name, need):
            if not isinstance(need, SeveralNeeds):
                return view(name, True)
            return CacheView("several", True,
                             parts=[several((name, j), part) for j, part in enumerate(need.parts)])

        for i, need in enumerate(needs):
            if isinstance(need, SeveralNeeds):
                self._views[i] = several(i, need)
                continue
            self._views[i] = view(cache_of[i] if cache_of[i] is not None else i,
                                  cache_of[i] is None)

    # ---- what the model sees ---------------------------------------------------------

    def views(self) -> List[Optional[CacheView]]:
        return self._views

    def bytes_per_token(self) -> int:
        """Bytes of keys and values one cached token takes over all groups."""
        size = torch.empty((), dtype=self.dtype).element_size()
        return sum(len(g.calls) * g.need.num_kv_heads * (g.need.head_dim + g.need.value_dim) * size
                   // g.need.every for g in self.groups)

    # ---- requests --------------------------------------------------------------------

    def has(self, req) -> bool:
        return req in self.requests

    def can_add(self) -> bool:
        return self.slots.available > 0

    def add(self, req) -> RequestCache:
        if req in self.requests:
            raise CacheError(f"request {req!r} is already live")
        rc = RequestCache(slot=self.slots.alloc(),
                          tables=[PageTable() for _ in self.groups],
                          first_live=[0 for _ in self.groups])
        # The slot's records read as zero for the new request, whoever held it before: a
        # mixer's state "before position 0" is part of this contract, not of each mixer.
        # (In stream order this comes after every step of the slot's previous holder.)
        for block in self._state_blocks:
            block[:, rc.slot].zero_()
        self.requests[req] = rc
        return rc

    def _first_needed_page(self, grp: Group, computed: int) -> int:
        """First page a query at position >= `computed` can still read."""
        lowest_key = 0
        if grp.need.window is not None:
            lowest_key = max(0, computed - grp.need.window + 1)
        if grp.need.chunk is not None:
            # the chunk of the next query begins here; earlier chunks are never read again
            lowest_key = max(lowest_key, computed // grp.need.chunk * grp.need.chunk)
        if grp.need.block is not None:
            # the block that the next query's token belongs to is read once more when complete
            lowest_key = min(lowest_key, computed // grp.need.block * grp.need.block)
        return grp.need.rows(lowest_key) // self.page_size

    def pages_for(self, grp: Group, tokens: int) -> int:
        """Block-table entries of `grp` that cover positions [0, tokens)."""
        return -(-grp.need.rows(tokens) // self.page_size)

    def room(self, req=None) -> int:
        """The most positions `req` (None: a new request) could cover with the free pages."""
        rc = self.requests.get(req) if req is not None else None
        most = 1 << 30
        for gi, grp in enumerate(self.groups):
            have = len(rc.tables[gi]) if rc else 0
            rows = (have + grp.pool.available) * self.page_size
            most = min(most, rows * grp.need.every + grp.need.every - 1)
        return most

    def pages_needed(self, req, total_tokens: int) -> List[int]:
        """Pages each group would have to hand out to cover positions
        [0, total_tokens) of `req` (which may not be live yet)."""
        rc = self.requests.get(req)
        out = []
        for gi, grp in enumerate(self.groups):
            have = len(rc.tables[gi]) if rc else 0
            out.append(max(0, self.pages_for(grp, total_tokens) - have))
        return out

    def can_reserve(self, req, total_tokens: int) -> bool:
        return all(n <= g.pool.available
                   for n, g in zip(self.pages_needed(req, total_tokens), self.groups))

    def reserve(self, req, total_tokens: int) -> bool:
        """Hand out pages so that positions [0, total_tokens) of `req` have a slot.
        All or nothing: returns False and changes nothing when a group lacks pages."""
        rc = self.requests[req]
        if total_tokens <= rc.tokens:
            return True
        want = [self.pages_for(grp, total_tokens) for grp in self.groups]
        if all(len(t) >= w for t, w in zip(rc.tables, want)):
            rc.tokens = total_tokens                 # room left in the last page
            return True
        if not self.can_reserve(req, total_tokens):
            return False
        for gi, grp in enumerate(self.groups):
            table = rc.tables[gi]
            while len(table) < want[gi]:
                table.append(grp.pool.alloc())
        rc.tokens = total_tokens
        return True

    def advance(self, req, computed: int) -> int:
        """Record that positions [0, computed) are written; give back the pages of
        windowed groups that no later query can see.  Returns how many were freed."""
        rc = self.requests[req]
        if computed < rc.computed:
            raise CacheError(f"request {req!r}: cannot move back from {rc.computed} "
                             f"to {computed} tokens")
        if computed > rc.tokens:
            raise CacheError(f"request {req!r}: {computed} tokens written but only "
                             f"{rc.tokens} reserved")
        rc.computed = computed
        freed = 0
        for gi, grp in enumerate(self.groups):
            first = min(self._first_needed_page(grp, computed), len(rc.tables[gi]))
            # the pages of positions that stay visible for good are never given back before the end
            kept = -(-grp.need.rows(grp.need.keep_first) // self.page_size)
            for p in range(max(rc.first_live[gi], kept), first):
                grp.pool.free(rc.tables[gi][p])
                rc.tables[gi][p] = -1
                freed += 1
            rc.first_live[gi] = max(rc.first_live[gi], first)
        return freed

    def free(self, req) -> None:
        """Give back everything `req` holds."""
        rc = self.requests.pop(req, None)
        if rc is None:
            raise CacheError(f"request {req!r} is not live")
        for gi, grp in enumerate(self.groups):
            for page in rc.tables[gi]:
                if page >= 0:
                    grp.pool.free(page)
        self.slots.free(rc.slot)

    # ---- checks ----------------------------------------------------------------------

    def check(self) -> None:
        """No page lost, none held twice: every page is on the free list or in exactly
        one block table; likewise the slots."""
        for gi, grp in enumerate(self.groups):
            held = [p for rc in self.requests.values() for p in rc.tables[gi] if p >= 0]
            if len(held) != len(set(held)):
                raise CacheError(f"group {gi}: a page is in two block tables")
            if len(held) != grp.pool.in_use:
                raise CacheError(f"group {gi}: {grp.pool.in_use} pages are out but block "
                                 f"tables hold {len(held)}")
            for p in held:
                if not grp.pool.is_held(p):
                    raise CacheError(f"group {gi}: page {p} is in a block table and on "
                                     f"the free list")
        slots = [rc.slot for rc in self.requests.values()]
        if len(slots) != len(set(slots)) or len(slots) != self.slots.in_use:
            raise CacheError("state slots and live requests disagree")
