"""The cache of a model: per-sequence slots, paged keys and values in groups of
layers with equal needs, and a per-sequence state area of fixed size.

What a run of a layer needs is said by its mixer (a :class:`KVRequest`, a :class:`RowsRequest`, a
:class:`StateRequest`, a tuple of those for several blocks, a :class:`BundleRequest` of such requests for a
mixer made of several mixers, or nothing). Runs with the same key/value geometry and
window share one :class:`KVGroup` — one storage tensor and one page map —
so layers that keep all keys and layers that keep a window of them have storage
of their own. State requests get one row per slot each, zeroed when the slot is
taken (a recurrent state must not start from a former sequence's values; key and
value pages need no clearing because lengths mask them).

Reference: inference/KVCache.java:87-136 (one array per layer and request),
inference/InferenceState.java:24-58 (per-request buffers); the fixed-size states of
its recurrent architectures live in per-request objects too
(inference/Qwen35State.java:39-42).
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch

from ..errors import CacheError, CacheFull
from .pages import PAGE_SIZE, FreeList, PageMap


@dataclass(frozen=True)
class KVRequest:
    """Keys and values of every position (or of a window of positions) of a sequence. ``keep_first``: with a window,
    the pages that hold a sequence's first so many positions are kept as well. ``chunk``: queries see keys of their own
    chunk of so many positions only (counted from the sequence's start), so pages of finished chunks go back."""
    num_kv_heads: int
    head_dim: int
    window: Optional[int] = None
    keep_first: int = 0
    chunk: Optional[int] = None


@dataclass(frozen=True)
class RowsRequest:
    """One row of ``width`` values for every position (or a window of positions) of a sequence: what a
    mixer keeps that attends over something other than per-head keys and values (a shared latent, say)."""
    width: int
    window: Optional[int] = None


@dataclass(frozen=True)
class StateRequest:
    """A block of fixed shape per sequence, zero at the sequence's start."""
    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


def keeps_state(request) -> bool:
    """Whether a run with this request keeps a state that a step changes in place (running a step twice would change
    it twice), by itself or as a member of a bundle."""
    if isinstance(request, BundleRequest):
        return any(keeps_state(m) for m in request.members)
    return isinstance(request, StateRequest) or (isinstance(request, tuple) and bool(request))


@dataclass(frozen=True)
class BundleRequest:
    """What a run keeps when its mixer is made of several mixers that each keep something: one request (a paged one, a
    state block, a tuple of state blocks, or None) per member, in the members' order."""
    members: Tuple[object, ...]


class BundleView:
    """The views of a :class:`BundleRequest`'s members, in order (None for a member that keeps nothing)."""

    def __init__(self, members: Sequence[object]):
        self.members = list(members)


class KVGroup:
    """Storage of the runs that share one paged request.

    ``storage[i]`` is the tensor of the i-th run of the group: for a :class:`KVRequest`
    [num_pages, 2 (keys, values), kv heads, PAGE_SIZE, head_dim], for a :class:`RowsRequest`
    [num_pages, PAGE_SIZE, width].
    """

    def __init__(self, request, runs: Sequence[int], num_pages: int, dtype: torch.dtype, device):
        self.request = request
        self.runs = list(runs)
        self.pages = PageMap(num_pages, window=request.window, keep_first=getattr(request, "keep_first", 0),
                             chunk=getattr(request, "chunk", None))
        if isinstance(request, RowsRequest):
            page_shape = (PAGE_SIZE, request.width)
        else:
            page_shape = (2, request.num_kv_heads, PAGE_SIZE, request.head_dim)
        # zeros once, so that stale rows are always finite; never cleared again
        self.storage = torch.zeros((len(self.runs), num_pages) + page_shape, dtype=dtype, device=device)

    def bytes_per_token(self) -> int:
        r = self.request
        per = r.width if isinstance(r, RowsRequest) else 2 * r.num_kv_heads * r.head_dim
        return len(self.runs) * per * self.storage.element_size()

    def view_of(self, run: int) -> torch.Tensor:
        return self.storage[self.runs.index(run)]


class KVView:
    """What an attention run sees of the cache: its storage and its group's index."""

    def __init__(self, group_index: int, pages: torch.Tensor):
        self.group_index = group_index
        self.pages = pages


class StateView:
    """What a run with fixed-size state sees: one row per slot (``rows``); a run that asked for several blocks
    (a tuple of :class:`StateRequest`) finds them all in ``blocks``, in the order it asked."""

    def __init__(self, rows: torch.Tensor, blocks: Optional[Sequence[torch.Tensor]] = None):
        self.rows = rows
        self.blocks = list(blocks) if blocks is not None else [rows]


class SequenceCache:
    def __init__(self, requests: Sequence[object], *, max_tokens: int, max_slots: Optional[int], kv_dtype: torch.dtype,
                 device):
        """``requests[i]``: what run i of the schedule keeps (a paged request, state requests, a bundle of those, or None)."""
        if max_tokens <= 0:
            raise CacheError(f"max_tokens must be positive, got {max_tokens}")
        self.device = device
        self.num_pages = -(-max_tokens // PAGE_SIZE)
        self.max_slots = max_slots if max_slots is not None else self.num_pages
        if self.max_slots <= 0:
            raise CacheError(f"max_slots must be positive, got {self.max_slots}")
        self.slots = FreeList(self.max_slots, "slot")
        self._length: Dict[int, int] = {}
        self.groups: List[KVGroup] = []
        self._views: List[object] = [None] * len(requests)
        # every paged request (a run's own, or a member's of a run's bundle) is a leaf with a key of its own
        leaves: List[Tuple[object, object]] = []

        def paged_leaves(key, req):
            if isinstance(req, (KVRequest, RowsRequest)):
                leaves.append((key, req))
            elif isinstance(req, BundleRequest):
                for i, member in enumerate(req.members):
                    paged_leaves(key + (i,), member)

        for run, req in enumerate(requests):
            paged_leaves((run,), req)
        by_request: Dict[object, List[object]] = {}
        for key, req in leaves:
            by_request.setdefault(req, []).append(key)
        paged_views: Dict[object, KVView] = {}
        for req, keys in by_request.items():
            group = KVGroup(req, keys, self.num_pages, kv_dtype, device)
            for key in keys:
                paged_views[key] = KVView(len(self.groups), group.view_of(key))
            self.groups.append(group)
        self._state_rows: List[torch.Tensor] = []

        def make_view(key, req):
            if req is None:
                return None
            if isinstance(req, (KVRequest, RowsRequest)):
                return paged_views[key]
            if isinstance(req, BundleRequest):
                return BundleView([make_view(key + (i,), member) for i, member in enumerate(req.members)])
            if isinstance(req, StateRequest):
                req = (req,)
            if isinstance(req, tuple) and req and all(isinstance(r, StateRequest) for r in req):
                blocks = [torch.zeros((self.max_slots,) + tuple(r.shape), dtype=r.dtype, device=device) for r in req]
                self._state_rows.extend(blocks)
                return StateView(blocks[0], blocks)
            raise CacheError(f"run {key[0]}: unknown cache request {req!r}")

        for run, req in enumerate(requests):
            self._views[run] = make_view((run,), req)

    # ------------------------------------------------------------------ slots
    def acquire(self) -> int:
        slot = self.slots.take()
        self._length[slot] = 0
        for group in self.groups:
            group.pages.open(slot)
        for rows in self._state_rows:
            rows[slot].zero_()
        return slot

    def release(self, slot: int) -> None:
        if not self.slots.is_held(slot):
            raise CacheError(f"slot {slot} is not held (freed twice?)")
        for group in self.groups:
            group.pages.close(slot)
        del self._length[slot]
        self.slots.give_back(slot)

    def length(self, slot: int) -> int:
        try:
            return self._length[slot]
        except KeyError:
            raise CacheError(f"slot {slot} is not held") from None

    def view(self, run: int):
        return self._views[run]

    # ------------------------------------------------------------------ a step
    def reserve(self, slots: Sequence[int], new_tokens: Sequence[int]) -> None:
        """Give every slot the pages its new tokens need; nothing changes if they do not all fit."""
        seen = set()
        for slot in slots:
            if slot in seen:
                raise CacheError(f"slot {slot} appears twice in one step")
            seen.add(slot)
            self.length(slot)
        for group in self.groups:
            need = sum(group.pages.pages_needed(s, self._length[s] + n) for s, n in zip(slots, new_tokens))
            if need > group.pages.pool.num_free:
                raise CacheFull(
                    f"the cache is full: this step needs {need} more page(s) of {PAGE_SIZE} positions, "
                    f"{group.pages.pool.num_free} of {group.pages.pool.count} are free")
        for group in self.groups:
            for s, n in zip(slots, new_tokens):
                group.pages.extend(s, self._length[s] + n)

    def reserve_up_to(self, slots: Sequence[int], lengths: Sequence[int]) -> None:
        """Pages for every slot up to the given total length, ahead of the steps that fill them."""
        self.reserve(slots, [max(0, n - self.length(s)) for s, n in zip(slots, lengths)])

    def commit(self, slots: Sequence[int], new_tokens: Sequence[int]) -> None:
        """The step ran: lengths grow, pages behind a window go back."""
        for s, n in zip(slots, new_tokens):
            self._length[s] += n
            for group in self.groups:
                group.pages.trim(s, self._length[s])

    def page_tables(self, slots: Sequence[int]) -> List[List[List[int]]]:
        """Per group, per slot of the step: page id of each block of positions."""
        return [[group.pages.table(s) for s in slots] for group in self.groups]

    # ------------------------------------------------------------------ reporting
    def memory_bytes(self) -> int:
        total = sum(g.storage.numel() * g.storage.element_size() for g in self.groups)
        total += sum(r.numel() * r.element_size() for r in self._state_rows)
        return total

    def free_pages(self) -> List[int]:
        return [g.pages.pool.num_free for g in self.groups]
