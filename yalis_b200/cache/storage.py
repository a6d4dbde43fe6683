"""Device memory behind the cache manager: page pools and per-request state.

For every schedule entry of a model the mixer's ``cache_request()`` says what
it keeps: keys and values in pages (``PagedKV``), a fixed-size state per request
(``SlotState``), or nothing.  Paged entries with the same retention rule (all
keys, or a window of W) form one *page group*: they share block tables, so one
page id means the same token range in each of their pools, and every group has
pages of its own.  Entries that keep one row per block of P tokens
(``PagedKV.pool``) form groups of their own too: a page holds as many rows, which
stand for P times as many tokens, and that is the page size the manager counts in.
Each paged entry owns two pools
``[num_pages, kv_heads, page_size, head_dim]`` (a KV head's tokens of one page
are contiguous, so the attention kernels stream whole pages per head); the
reference lays a page out as ``[page, kv_heads, head_dim]`` per token
(yalis/external/model.py:620-627).  Pools are never cleared: what a request can
see is decided by its length and its block table only.
"""

from __future__ import annotations

from typing import Dict, List, Optional

import torch

from collections.abc import Mapping

from yalis_b200.parts.base import PagedKV, PagedKVCache, SlotState, SlotStateCache, cache_leaves
from .manager import PageGroup


def group_name(request: PagedKV) -> str:
    """Paged entries with the same retention rule share block tables (a page id means the same token range
    in each of their pools); the rule is all a group is known by."""
    name = "kv_all" if request.window is None else f"kv_window_{request.window}"
    return name if request.pool == 1 else f"{name}_pool_{request.pool}"


def group_page_bytes(requests: List[Optional[object]], cache_of: List[Optional[int]], page_size: int,
                     element_size: int) -> Dict[str, int]:
    """Bytes that one page id of each group stands for: the K and V pages of every schedule entry of the group
    that keeps a cache of its own (of a group with a row per P tokens, the P-th part: it has so many fewer pages)."""
    out: Dict[str, int] = {}
    for top, src in zip(requests, cache_of):
        for req in cache_leaves(top):
            if isinstance(req, PagedKV) and src is None:
                name = group_name(req)
                out[name] = out.get(name, 0) + -(-req.num_kv_heads * page_size * (req.head_dim + req.value_dim) * element_size // req.pool)
    return out


def window_group_pages(window: int, page_size: int, max_slots: int, step_tokens: int) -> int:
    """Pages a group with a window can have in use at once: per request the window, the tokens of the step that
    is running (their pages are mapped before the step and those behind the window returned after it) and the
    two partly used pages at the ends."""
    return max_slots * (-(-(window + step_tokens) // page_size) + 2)


def plan_groups(requests: List[Optional[object]], page_size: int, num_pages: int, max_context: int,
                max_slots: Optional[int] = None, step_tokens: Optional[int] = None) -> List[PageGroup]:
    """One page group per distinct retention rule among the paged requests.  ``num_pages`` is the pool of a
    group that keeps every key; a group with a window gets no more pages than it can ever use
    (``window_group_pages``) when ``max_slots`` and ``step_tokens`` are known; a group with a row per P tokens gets the
    P-th part, and a page more per request."""
    groups: Dict[str, PageGroup] = {}
    for r in (leaf for top in requests for leaf in cache_leaves(top)):
        if isinstance(r, PagedKV):
            name = group_name(r)
            if name not in groups:
                pages = num_pages
                if r.window is not None and max_slots is not None and step_tokens is not None:
                    pages = min(pages, window_group_pages(r.window, page_size, max_slots, min(step_tokens, max_context)))
                if r.pool > 1 and max_slots is not None:
                    pages = min(pages, -(-pages // r.pool) + max_slots)
                covered = page_size * r.pool          # tokens that a page stands for
                groups[name] = PageGroup(name, covered, pages, r.window, -(-max_context // covered))
    return list(groups.values())


class CacheStorage:
    """Allocates what every schedule entry asked for and hands out the per-entry views."""

    def __init__(self, requests: List[Optional[object]], cache_of: List[Optional[int]], groups: List[PageGroup],
                 max_slots: int, device, dtype: torch.dtype):
        self._by_name = {g.name: g for g in groups}
        self._max_slots, self._device, self._dtype = max_slots, device, dtype
        self.entries: List[Optional[object]] = []
        self.state_tensors: List[torch.Tensor] = []
        self.bytes = 0
        for i, (req, src) in enumerate(zip(requests, cache_of)):
            if src is not None:
                self.entries.append(self._reader(i, src, req, self.entries[src]))
            else:
                self.entries.append(self._allocate(i, req))

    def _reader(self, i: int, src: int, req, own):
        """The cache of entry ``src`` as entry ``i`` may use it: read, never written."""
        if isinstance(own, dict):
            if not isinstance(req, Mapping) or set(req) != set(own):
                raise ValueError(f"schedule entry {i} cannot read the cache of entry {src}: they keep different things")
            return {name: self._reader(i, src, req[name], own[name]) for name in own}
        if isinstance(own, PagedKVCache):
            if not isinstance(req, PagedKV) or (req.num_kv_heads, req.head_dim, req.value_dim) != (own.k.shape[1], own.k.shape[3], own.v.shape[3]):
                raise ValueError(f"schedule entry {i} cannot read the cache of entry {src}: shapes differ")
            return PagedKVCache(own.k, own.v, own.group, writable=False)
        if isinstance(own, SlotStateCache):
            return SlotStateCache(own.state, writable=False)
        raise ValueError(f"schedule entry {i} reads the cache of entry {src}, which keeps none")

    def _allocate(self, i: int, req):
        if req is None:
            return None
        if isinstance(req, Mapping):
            return {name: self._allocate(i, sub) for name, sub in req.items()}
        if isinstance(req, PagedKV):
            g = self._by_name[group_name(req)]
            rows = g.page_size // req.pool
            k = torch.empty((g.num_pages, req.num_kv_heads, rows, req.head_dim), dtype=self._dtype, device=self._device)
            v = torch.empty((g.num_pages, req.num_kv_heads, rows, req.value_dim), dtype=self._dtype, device=self._device)
            self.bytes += k.numel() * k.element_size() + v.numel() * v.element_size()
            return PagedKVCache(k, v, g.name)
        if isinstance(req, SlotState):
            # one row more than there are slots: the row that padding rows of a recorded step point to
            st = torch.zeros((self._max_slots + 1,) + tuple(req.shape), dtype=req.dtype, device=self._device)
            self.bytes += st.numel() * st.element_size()
            self.state_tensors.append(st)
            return SlotStateCache(st)
        raise TypeError(f"schedule entry {i}: unknown cache request {req!r}")

    def reset_slot(self, slot: int) -> None:
        """Zero the per-request state of a newly admitted request."""
        for st in self.state_tensors:
            st[slot].zero_()

    def snapshot_state(self) -> List[torch.Tensor]:
        """Copies of all per-request state (for a trial run whose effects must not stay)."""
        return [st.clone() for st in self.state_tensors]

    def restore_state(self, saved: List[torch.Tensor]) -> None:
        for st, old in zip(self.state_tensors, saved):
            st.copy_(old)
