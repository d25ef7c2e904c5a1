"""The cache on the device: paged keys and values per group of layers, and a
fixed-size state row per slot.

Each mixer says what it needs of the cache (`KVRequirement`: all keys or a
window of them; `StateRequirement`: a tensor of fixed shape per sequence).
Cache entries with the same key/value needs form a *group* with storage, a
page pool and a block table of its own; within a group a page id means the
same page in every layer, so one table row serves all its layers.  Lengths
live on the host; the step function writes per-token positions and slots for
the kernels.

A mixer that reads the means of whole blocks of keys and values behind a
window (`KVRequirement.mean_block`) gets a second group with a row per block:
the window's pages come back as they fall out of it, the block rows stay.

Pools are `[n_pages, n_kv_heads, page_size, head_dim]` per layer, keys and
values apart (upstream: src/kvcache.h:49-50, page size fixed to 32 at
kvcache.h:7, one table per layer).  Pools start zeroed and only ever hold
finite numbers, so a kernel may read a page's unused rows and mask them.
"""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence, Union

import numpy as np
import torch

from .allocator import CacheError, GroupTable, SlotAllocator

TOKEN_UNIT = 64     # capacities are counted per sequence in units of this many tokens


@dataclass(frozen=True)
class KVRequirement:
    n_kv_heads: int
    head_dim: int
    window: Optional[int] = None      # None: every earlier key; w: the last w keys
    planes: int = 2                   # 2: keys and values apart; 1: one row per position (a latent that keys
                                      # and values are both made from), and the view's v_pool is its k_pool
    value_heads: Optional[int] = None   # values of a shape of their own (None: the keys' heads / head_dim):
    value_dim: Optional[int] = None     # the value pool is then [n_pages, value_heads, page_size, value_dim]
    mean_block: Optional[int] = None    # P: beside the tokens' rows one row (key and value) for every whole block of P
                                        # positions, kept for the sequence's whole life on pages of its own
    keep_first: int = 0               # with a window: the first positions of a sequence stay beside it

    @property
    def value_shape(self) -> tuple:
        return (self.value_heads or self.n_kv_heads, self.value_dim or self.head_dim)


@dataclass(frozen=True)
class StateRequirement:
    shape: tuple
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class EntryRequirement:
    """A cache entry that holds both: paged keys and values, and a state row per slot (a mixer that runs an
    attention and a recurrence side by side, or an attention behind short convolutions)."""
    kv: Optional[KVRequirement] = None
    state: Optional[StateRequirement] = None


Requirement = Union[KVRequirement, StateRequirement, EntryRequirement, None]


def split_requirement(req) -> tuple:
    """(paged part, state part) of any requirement."""
    if isinstance(req, EntryRequirement):
        return req.kv, req.state
    if isinstance(req, KVRequirement):
        return req, None
    if isinstance(req, StateRequirement):
        return None, req
    if req is None:
        return None, None
    raise CacheError(f"unknown cache requirement {req!r}")


@dataclass
class MeansView:
    """The rows that stand for whole blocks of positions: row b of a sequence covers positions b block .. (b + 1) block - 1."""
    k_pool: torch.Tensor          # [n_pages, n_kv, rows, d]
    v_pool: torch.Tensor
    block_table: torch.Tensor     # int32 [max_slots, max_pages_per_seq]
    block: int


@dataclass
class KVView:
    """What a mixer gets for one cache entry in one step."""
    k_pool: torch.Tensor          # [n_pages, n_kv, page_size, d]
    v_pool: torch.Tensor
    block_table: torch.Tensor     # int32 [max_slots, max_pages_per_seq], -1 = no page
    page_size: int
    window: Optional[int]
    means: Optional[MeansView] = None


@dataclass
class EntryView:
    """Everything one cache entry holds: paged keys/values and/or a state tensor [max_slots, ...]."""
    kv: Optional[KVView] = None
    state: Optional[torch.Tensor] = None


def mean_page_rows(page_size: int, block: int) -> int:
    """Rows of a page of block rows: about as many positions as a page of tokens covers, but a power of two of at least
    8 rows (the pieces that the prompt kernel copies)."""
    rows = 8
    while rows * block < page_size:
        rows *= 2
    return rows


class _KVGroup:
    """`mean_block` P: a row for every whole block of P positions of a sequence (kept whatever the window is) instead of one
    for every position."""

    def __init__(self, req: KVRequirement, entries: list[int], n_pages: int, page_size: int, max_slots: int,
                 max_pages_per_seq: int, dtype: torch.dtype, device, mean_block: Optional[int] = None):
        self.req = req
        self.entries = entries
        self.stride = mean_block or 1                # positions a row stands for
        self.host = GroupTable(n_pages, page_size, max_slots, max_pages_per_seq, None if mean_block else req.window, 0 if mean_block else req.keep_first)
        if req.planes not in (1, 2):
            raise CacheError(f"a paged entry holds 1 or 2 rows per position, not {req.planes}")
        self.storage = self.k_storage = self.v_storage = None
        if req.value_shape == (req.n_kv_heads, req.head_dim) or req.planes == 1:
            self.storage = torch.zeros((len(entries), req.planes, n_pages, req.n_kv_heads, page_size, req.head_dim),
                                       dtype=dtype, device=device)
        else:                                    # keys and values of different shapes: a tensor each
            vh, vd = req.value_shape
            self.k_storage = torch.zeros((len(entries), n_pages, req.n_kv_heads, page_size, req.head_dim),
                                         dtype=dtype, device=device)
            self.v_storage = torch.zeros((len(entries), n_pages, vh, page_size, vd), dtype=dtype, device=device)
        self.table = torch.full((max_slots, max_pages_per_seq), -1, dtype=torch.int32, device=device)

    def pools(self, i: int) -> tuple:
        if self.storage is not None:
            return self.storage[i, 0], self.storage[i, self.req.planes - 1]
        return self.k_storage[i], self.v_storage[i]

    def bytes_per_token(self) -> int:
        vh, vd = self.req.value_shape
        per = self.req.n_kv_heads * self.req.head_dim + (vh * vd if self.req.planes == 2 else 0)
        size = (self.storage if self.storage is not None else self.k_storage).element_size()
        return -(-len(self.entries) * per * size // self.stride)

    def upload(self) -> None:
        if not self.host.dirty:
            return
        rows = sorted(self.host.dirty)
        self.host.dirty.clear()
        idx = torch.as_tensor(rows, dtype=torch.long)
        src = torch.from_numpy(self.host.table[rows])
        if self.table.is_cuda:                   # pinned, so that neither copy waits for the steps in flight
            idx, src = idx.pin_memory(), src.pin_memory()
        self.table.index_copy_(0, idx.to(self.table.device, non_blocking=True),
                               src.to(self.table.device, non_blocking=True))


class PagedCache:
    """Slots, pages and state for one model.

    `requirements[e]` is what cache entry `e` needs (None for a mixer that keeps nothing).
    `max_tokens` is the most tokens that live sequences hold at any time, each sequence counted
    in units of 64 tokens."""

    def __init__(self, requirements: Sequence[Requirement], max_tokens: int, max_positions: int,
                 dtype: torch.dtype, device, page_size: int = 64, max_slots: Optional[int] = None):
        if page_size <= 0:
            raise CacheError(f"page_size must be positive, not {page_size}")
        if max_tokens <= 0:
            raise CacheError(f"max_tokens must be positive, not {max_tokens}")
        units = -(-max_tokens // TOKEN_UNIT)
        self.page_size = page_size
        self.max_tokens = units * TOKEN_UNIT
        self.max_positions = max_positions
        self.max_slots = max_slots or units
        self.n_pages = units * (-(-TOKEN_UNIT // page_size)) if page_size <= TOKEN_UNIT else units
        longest = min(max_positions, self.max_tokens)
        self.max_pages_per_seq = -(-longest // page_size)
        self._longest = longest
        self.dtype, self.device = dtype, torch.device(device)
        self.slots = SlotAllocator(self.max_slots)
        self.lengths = np.zeros(self.max_slots, dtype=np.int64)

        self.groups: list[_KVGroup] = []
        self._kv_of_entry: dict[int, tuple[_KVGroup, int]] = {}
        self._means_of_entry: dict[int, _KVGroup] = {}        # same place in the group as the entry's tokens
        self._state_of_entry: dict[int, torch.Tensor] = {}
        by_req: dict[KVRequirement, list[int]] = {}
        for e, req in enumerate(requirements):
            kv_req, state_req = split_requirement(req)
            if kv_req is not None:
                by_req.setdefault(kv_req, []).append(e)
            if state_req is not None:
                # one row per slot and a spare last row: a padding row of a recorded step carries slot -1,
                # which as an index is that spare, so it reads and writes nothing a sequence owns
                self._state_of_entry[e] = torch.zeros((self.max_slots + 1, *state_req.shape), dtype=state_req.dtype,
                                                      device=self.device)
        for req, entries in by_req.items():
            g = _KVGroup(req, entries, self.n_pages, page_size, self.max_slots, self.max_pages_per_seq,
                         dtype, self.device)
            self.groups.append(g)
            for i, e in enumerate(entries):
                self._kv_of_entry[e] = (g, i)
            if req.mean_block:
                means = self._means_group(req, entries, units)
                self.groups.append(means)
                for e in entries:
                    self._means_of_entry[e] = means
        # set by the kernels when an index they were given is out of range (0 = all well)
        self.status = torch.zeros(1, dtype=torch.int32, device=self.device)

    def _means_group(self, req: KVRequirement, entries: list[int], units: int) -> _KVGroup:
        if req.mean_block < 1 or req.planes != 2:
            raise CacheError(f"rows for blocks of {req.mean_block} positions of an entry with {req.planes} rows per position")
        if req.window is not None and req.window < req.mean_block:
            raise CacheError(f"blocks of {req.mean_block} positions are not whole inside a window of {req.window}")
        rows = mean_page_rows(self.page_size, req.mean_block)
        covers = rows * req.mean_block                        # positions a page stands for
        # a sequence of u units of TOKEN_UNIT positions needs at most u times this many pages; and no more than one
        # part-filled page per slot beside the whole ones
        n_pages = min(units * (-(-TOKEN_UNIT // covers) if covers <= TOKEN_UNIT else 1),
                      self.max_slots + self.max_tokens // covers)
        return _KVGroup(req, entries, n_pages, rows, self.max_slots, -(-self._longest // covers), self.dtype, self.device,
                        mean_block=req.mean_block)

    # ---- slots -------------------------------------------------------------------
    def alloc_slot(self) -> int:
        s = self.slots.alloc()
        self.lengths[s] = 0
        for st in self._state_of_entry.values():
            st[s].zero_()
        return s

    def free_slot(self, slot: int) -> None:
        self.slots.free(slot)
        for g in self.groups:
            g.host.release(slot)
        self.lengths[slot] = 0

    def length(self, slot: int) -> int:
        return int(self.lengths[slot])

    @property
    def state_bytes_per_slot(self) -> int:
        return sum(int(np.prod(st.shape[1:])) * st.element_size() for st in self._state_of_entry.values())

    # ---- one step ------------------------------------------------------------------
    def prepare(self, slots: Sequence[int], n_new: Sequence[int]) -> None:
        """Give every listed slot room for `n_new` more positions, or raise before anything changed."""
        seen = set()
        for s, n in zip(slots, n_new):
            if not self.slots.is_live(s):
                raise CacheError(f"slot {s} is not in use")
            if s in seen:
                raise CacheError(f"slot {s} appears twice in one step")
            seen.add(s)
            if n < 0:
                raise CacheError("a step cannot bring a negative number of tokens")
            if self.lengths[s] + n > self.max_positions:
                raise CacheError(f"slot {s} would reach {self.lengths[s] + n} positions; the model's "
                                 f"limit is {self.max_positions}")
            if -(-(int(self.lengths[s]) + n) // self.page_size) > self.max_pages_per_seq:
                raise CacheError(f"slot {s} would reach {self.lengths[s] + n} positions; the cache was "
                                 f"sized for {self.max_pages_per_seq * self.page_size} per sequence")
        for g in self.groups:
            need = sum(g.host.pages_needed(s, (int(self.lengths[s]) + n) // g.stride) for s, n in zip(slots, n_new))
            if need > g.host.pool.n_free:
                raise CacheError(f"the cache is full: this step needs {need} more pages of "
                                 f"{g.host.page_size * g.stride} tokens, {g.host.pool.n_free} of {g.host.pool.n_pages} are free")
        for g in self.groups:
            for s, n in zip(slots, n_new):
                g.host.reserve(s, (int(self.lengths[s]) + n) // g.stride)
            g.upload()

    def commit(self, slots: Sequence[int], n_new: Sequence[int]) -> None:
        """The step ran: lengths grow, windowed groups drop what no later query can see."""
        for s, n in zip(slots, n_new):
            self.lengths[s] += n
            for g in self.groups:
                g.host.trim(s, int(self.lengths[s]))

    # ---- views -----------------------------------------------------------------------
    def kv_view(self, entry: int) -> Optional[KVView]:
        if entry not in self._kv_of_entry:
            return None
        g, i = self._kv_of_entry[entry]
        m = self._means_of_entry.get(entry)
        means = MeansView(*m.pools(i), m.table, m.stride) if m is not None else None
        return KVView(*g.pools(i), g.table, self.page_size, g.req.window, means)

    def state_view(self, entry: int) -> Optional[torch.Tensor]:
        return self._state_of_entry.get(entry)

    def view(self, entry: int, kv_entry: Optional[int] = None) -> EntryView:
        """What a layer run sees: the state of `entry` and the paged keys and values of `kv_entry` (another entry,
        for a layer that reads the keys and values another layer wrote), or of `entry` itself."""
        return EntryView(self.kv_view(entry if kv_entry is None else kv_entry), self.state_view(entry))

    def check_status(self) -> None:
        code = int(self.status.item())
        if code:
            self.status.zero_()
            raise CacheError(f"a kernel was given an index outside the cache (code {code}): "
                             "1 position beyond the block table, 2/5 unmapped page, 3 position beyond "
                             "the rotary table, 4 query position beyond the block table")

    def bytes_per_token(self) -> int:
        return sum(g.bytes_per_token() for g in self.groups)
