"""The cache: a slot per sequence, paged keys and values per layer group,
and fixed-size per-sequence state.

* A *slot* belongs to one live sequence and carries its length.  Slots are
  handed back when a sequence ends and are used again without clearing:
  what is valid is known from the length alone, as in the reference
  (src/model/cache.rs:301-310, where ``clear`` only resets the position).
* Keys and values live in *pages* of ``page_tokens`` positions.  Layers
  with the same need (kv heads, head size, window) form a *group* with its
  own pool of pages and its own page table; a sequence's pages are taken
  from the pool as it grows.  A group whose layers see all keys keeps every
  position; a group with a window keeps a ring of the last
  ``ring_tokens`` positions (position p lives in cell p % ring_tokens): the
  window plus room for the longest step that continues a sequence
  (``max_continuation`` positions; by default one page more than the window).
* A group whose need names ``pool`` = P also keeps one *cell* per block of P positions
  (positions bP .. bP + P - 1; the mixer writes a block's cell in the step that brings the
  block's last position): a second paged store whose "position" b is block b and which
  never wraps.  Its ring then keeps max(window, P) positions, so that a block's positions
  are still there when its last one arrives.
* *State* is a fixed-size tensor per slot and schedule entry for mixers
  that carry a recurrent state instead of keys; it is zeroed when the slot
  is acquired.  (The attention mixer needs none.)  A part at a mixer's input (a short
  convolution) has a second one beside the mixer's, ``CacheNeed.inputs``.
* A group whose need names ``keep_first`` = K (with a window) keeps the sequence's first K
  positions for good: they lie in whole pages of their own ahead of the ring
  (``fixed_tokens`` positions, K rounded up to pages), which nothing overwrites; position
  p >= fixed_tokens lives in cell fixed_tokens + (p - fixed_tokens) % ring_tokens.

The reference keeps one dense [max_seq_len, kv_dim] buffer per layer and a
single position counter (src/model/cache.rs:23-43,77-112); its errors for
overflow and bad indices (:178-200,218-229) have their counterparts here.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, List, Optional, Sequence, Tuple

import torch


class CacheError(RuntimeError):
    pass


STATE_BUDGET = 24 << 30     # bytes of per-slot state a cache sized by default holds at most
MIN_SLOTS = 16


def _count(shape) -> int:
    n = 1
    for s in shape:
        n *= int(s)
    return n


class CacheFull(CacheError):
    """No free page (or slot) is left for what a step needs."""


class ContextOverflow(CacheError):
    """A sequence would grow beyond the engine's maximum length."""


@dataclass(frozen=True)
class KVNeed:
    """Per-position keys and values: what an attention-like mixer declares."""

    n_kv_heads: int
    head_dim: int            # width of a key
    window: int = 0          # 0: every earlier position stays visible
    value_dim: int = 0       # width of a value; 0: the same as a key
    # a value is (the leading part of) its key's cell: no pool of values is kept
    values_in_keys: bool = False
    # P > 0: beside the positions, one key cell and one value cell per block of P positions
    pool: int = 0
    # C > 0: a position is only ever read by the later positions of its own chunk of C (a mask
    # of chunks); every position is kept all the same, since a run that reads this cache may
    # cut its chunks elsewhere
    chunk: int = 0
    # K > 0 (with a window): the sequence's first K positions stay visible for good
    keep_first: int = 0

    @property
    def v_dim(self) -> int:
        return self.value_dim or self.head_dim


@dataclass(frozen=True)
class StateNeed:
    """Fixed-size per-sequence state: what a recurrent mixer declares."""

    shape: Tuple[int, ...]
    dtype: torch.dtype = torch.float32


@dataclass(frozen=True)
class CacheNeed:
    kv: Optional[KVNeed] = None
    state: Optional[StateNeed] = None
    # state of the part at the mixer's input, apart from the mixer's own
    inputs: Optional[StateNeed] = None


class PagePool:
    """Free-list of page numbers with ownership checks."""

    def __init__(self, n_pages: int):
        self.n_pages = n_pages
        self._free: List[int] = list(range(n_pages - 1, -1, -1))
        self._held = [False] * n_pages

    @property
    def n_free(self) -> int:
        return len(self._free)

    def take(self, n: int) -> List[int]:
        if n > len(self._free):
            raise CacheFull(f"{n} pages wanted, {len(self._free)} of {self.n_pages} are free")
        out = [self._free.pop() for _ in range(n)]
        for p in out:
            if self._held[p]:
                raise CacheError(f"page {p} handed out twice")
            self._held[p] = True
        return out

    def give_back(self, pages: Sequence[int]) -> None:
        for p in pages:
            if not 0 <= p < self.n_pages or not self._held[p]:
                raise CacheError(f"page {p} freed but not held")
            self._held[p] = False
            self._free.append(p)


class BlockCells:
    """One key cell and one value cell per block of ``block`` positions, for the layers of one
    group: pages of ``page_tokens`` cells, a page table per slot, every block kept."""

    def __init__(self, need: "KVNeed", n_entries: int, total_tokens: int, max_slots: int,
                 max_seq_len: int, page_tokens: int, dtype: torch.dtype, device: torch.device):
        self.block = need.pool
        self.page_tokens = page_tokens
        self.pages_per_seq = max(1, -(-(max_seq_len // self.block) // page_tokens))
        # every sequence may hold one partly filled page of cells beside its share of the blocks
        n_pages = -(-(total_tokens // self.block) // page_tokens) + max_slots
        self.n_pages = min(n_pages, max_slots * self.pages_per_seq)
        self.pool = PagePool(self.n_pages)
        shape = (n_entries, self.n_pages, need.n_kv_heads, page_tokens)
        self.k = torch.zeros(shape + (need.head_dim,), dtype=dtype, device=device)
        self.v = torch.zeros(shape + (need.v_dim,), dtype=dtype, device=device)
        self.table_host = torch.zeros((max_slots, self.pages_per_seq), dtype=torch.int32)
        self.table = torch.zeros((max_slots, self.pages_per_seq), dtype=torch.int32, device=device)
        self.pages: List[List[int]] = [[] for _ in range(max_slots)]
        self.dirty = False

    def pages_for(self, length: int) -> int:
        """Pages of cells a sequence of ``length`` positions holds (whole blocks only)."""
        return min(-(-(length // self.block) // self.page_tokens), self.pages_per_seq)

    def bytes(self) -> int:
        return (self.k.numel() + self.v.numel()) * self.k.element_size()


class KVGroup:
    """Storage of the layers (schedule entries) that share one :class:`KVNeed`."""

    def __init__(self, need: KVNeed, entries: List[int], n_pages: int, max_slots: int,
                 max_seq_len: int, page_tokens: int, dtype: torch.dtype, device: torch.device,
                 max_continuation: Optional[int] = None):
        self.need = need
        self.entries = list(entries)
        self.page_tokens = page_tokens
        full_pages = -(-max_seq_len // page_tokens)
        # what a ring keeps behind a position: the window, and a whole block where blocks are pooled
        self.keep = max(need.window, need.pool) if need.window > 0 else 0
        if need.keep_first > 0 and (need.window <= 0 or need.pool > 0 or need.values_in_keys):
            raise CacheError("kept first positions go with a window, and without pooled blocks or shared cells")
        # whole pages ahead of the ring for the positions that are kept for good
        fixed_pages = -(-need.keep_first // page_tokens)
        if need.window <= 0:
            ring_pages = full_pages
        elif max_continuation is None:
            ring_pages = -(-self.keep // page_tokens) + 1
        else:
            # a step of c positions writes c - 1 cells ahead of what its first row still sees
            ring_pages = -(-(self.keep + max(1, max_continuation) - 1) // page_tokens)
        if fixed_pages + ring_pages >= full_pages:
            self.ring_tokens = self.fixed_tokens = 0          # never wraps
            self.pages_per_seq = full_pages
        else:
            self.ring_tokens = ring_pages * page_tokens
            self.fixed_tokens = fixed_pages * page_tokens
            self.pages_per_seq = fixed_pages + ring_pages
        self.n_pages = min(n_pages, max_slots * self.pages_per_seq)
        self.pool = PagePool(self.n_pages)
        shape = (len(entries), self.n_pages, need.n_kv_heads, page_tokens)
        # zeroed once: kernels that work on whole tiles of positions may load a
        # cell that is masked out, and its bits must at least be a number
        self.k = torch.zeros(shape + (need.head_dim,), dtype=dtype, device=device)
        self.v = self.k if need.values_in_keys else \
            torch.zeros(shape + (need.v_dim,), dtype=dtype, device=device)
        self.table_host = torch.zeros((max_slots, self.pages_per_seq), dtype=torch.int32)
        self.table = torch.zeros((max_slots, self.pages_per_seq), dtype=torch.int32, device=device)
        self.pages: List[List[int]] = [[] for _ in range(max_slots)]
        self.dirty = False
        self.cells: Optional[BlockCells] = None
        if need.pool > 0:
            if need.window <= 0 or need.values_in_keys:
                raise CacheError("pooled blocks go with a window and with values of their own")
            self.cells = BlockCells(need, len(entries), n_pages * page_tokens, max_slots,
                                    max_seq_len, page_tokens, dtype, device)

    def pages_for(self, length: int) -> int:
        """Pages a sequence of ``length`` positions holds in this group."""
        return min(-(-length // self.page_tokens), self.pages_per_seq)

    def max_step_tokens(self, start: Optional[int] = None) -> int:
        """The most positions one step may add to a sequence without overwriting a key
        that a row of the same step still sees: the ring's room beyond the window, which
        holds wherever the sequence stands; a sequence that holds ``start`` positions may
        also add whatever does not wrap around the ring."""
        if self.ring_tokens == 0:
            return 1 << 30
        room = self.ring_tokens - self.keep + 1
        return room if start is None else max(self.fixed_tokens + self.ring_tokens - start, room)

    def bytes(self) -> int:
        held = self.k.numel() + (0 if self.v is self.k else self.v.numel())
        return held * self.k.element_size() + (self.cells.bytes() if self.cells else 0)


class SequenceCache:
    def __init__(self, needs: Sequence[Optional[CacheNeed]], max_tokens: int, max_seq_len: int,
                 dtype: torch.dtype, device, page_tokens: int = 64,
                 max_slots: Optional[int] = None, max_continuation: Optional[int] = None,
                 named_state: Optional[Dict[str, StateNeed]] = None):
        """``named_state``: fixed-size per-slot state that belongs to no schedule entry
        (an embedding that remembers a sequence's last token), by name."""
        if page_tokens <= 0 or max_tokens <= 0 or max_seq_len <= 0:
            raise CacheError("page_tokens, max_tokens and max_seq_len must be positive")
        device = torch.device(device)
        self.page_tokens = page_tokens
        self.max_seq_len = max_seq_len
        self.device = device
        self.total_pages = -(-max_tokens // page_tokens)
        self.max_tokens = self.total_pages * page_tokens
        self.max_slots = max_slots or min(self.total_pages, 4096)
        if max_slots is None:
            # (state is held for every slot, live or not: where the caller names no number of
            # slots, no more of them than keep the state within STATE_BUDGET bytes)
            per_slot = sum(_count(st.shape) * torch.empty((), dtype=st.dtype).element_size()
                           for need in needs if need is not None
                           for st in (need.state, need.inputs) if st is not None)
            if per_slot * self.max_slots > STATE_BUDGET:
                self.max_slots = max(MIN_SLOTS, min(self.max_slots, STATE_BUDGET // per_slot))
        # groups of schedule entries with the same need
        by_need: Dict[KVNeed, List[int]] = {}
        for entry, need in enumerate(needs):
            if need is not None and need.kv is not None:
                by_need.setdefault(need.kv, []).append(entry)
        self.groups: List[KVGroup] = [
            KVGroup(kv, entries, self.total_pages, self.max_slots, max_seq_len, page_tokens,
                    dtype, device, max_continuation) for kv, entries in by_need.items()]
        # everything that hands out pages: the groups and their stores of block cells
        self._stores = list(self.groups) + [g.cells for g in self.groups if g.cells is not None]
        self._where: Dict[int, Tuple[int, int]] = {}
        for gi, g in enumerate(self.groups):
            for li, entry in enumerate(g.entries):
                self._where[entry] = (gi, li)
        def per_slot_state(st: StateNeed) -> torch.Tensor:
            return torch.zeros((self.max_slots,) + tuple(st.shape), dtype=st.dtype, device=device)
        self.state: Dict[int, torch.Tensor] = {}
        self.inputs: Dict[int, torch.Tensor] = {}
        for entry, need in enumerate(needs):
            if need is not None and need.state is not None:
                self.state[entry] = per_slot_state(need.state)
            if need is not None and need.inputs is not None:
                self.inputs[entry] = per_slot_state(need.inputs)
        self.named: Dict[str, torch.Tensor] = {
            name: torch.zeros((self.max_slots,) + tuple(need.shape), dtype=need.dtype, device=device)
            for name, need in (named_state or {}).items()}
        self._free_slots: List[int] = list(range(self.max_slots - 1, -1, -1))
        self._live = [False] * self.max_slots
        self.lengths = [0] * self.max_slots

    # ---- slots --------------------------------------------------------
    @property
    def n_free_slots(self) -> int:
        return len(self._free_slots)

    def acquire(self) -> int:
        if not self._free_slots:
            raise CacheFull(f"all {self.max_slots} slots are in use")
        s = self._free_slots.pop()
        if self._live[s]:
            raise CacheError(f"slot {s} handed out twice")
        self._live[s] = True
        self.lengths[s] = 0
        for t in list(self.state.values()) + list(self.inputs.values()) + list(self.named.values()):
            t[s].zero_()
        return s

    def release(self, slot: int) -> None:
        self._check_slot(slot)
        for g in self._stores:
            g.pool.give_back(g.pages[slot])
            g.pages[slot] = []
        self._live[slot] = False
        self.lengths[slot] = 0
        self._free_slots.append(slot)

    def _check_slot(self, slot: int) -> None:
        if not isinstance(slot, int) or not 0 <= slot < self.max_slots:
            raise CacheError(f"slot {slot!r} does not exist (0..{self.max_slots - 1})")
        if not self._live[slot]:
            raise CacheError(f"slot {slot} is not in use")

    def length(self, slot: int) -> int:
        self._check_slot(slot)
        return self.lengths[slot]

    def live_slots(self) -> List[int]:
        return [s for s, l in enumerate(self._live) if l]

    # ---- growth -------------------------------------------------------
    def reserve(self, grow: Sequence[Tuple[int, int]]) -> None:
        """Make room for ``n`` more positions in each ``(slot, n)``; either
        every sequence gets its pages or nothing changes."""
        plan = []
        wanted = [0] * len(self._stores)
        for slot, n in grow:
            self._check_slot(slot)
            new_len = self.lengths[slot] + n
            if n < 0 or new_len > self.max_seq_len:
                raise ContextOverflow(f"slot {slot}: {self.lengths[slot]} + {n} positions exceed "
                                      f"the maximum sequence length {self.max_seq_len}")
            for gi, g in enumerate(self._stores):
                extra = g.pages_for(new_len) - len(g.pages[slot])
                if extra > 0:
                    plan.append((gi, slot, extra))
                    wanted[gi] += extra
        for gi, g in enumerate(self._stores):
            if wanted[gi] > g.pool.n_free:
                raise CacheFull(f"the cache holds {self.max_tokens} positions; {wanted[gi]} more "
                                f"pages of {self.page_tokens} are needed and {g.pool.n_free} are free")
        for gi, slot, extra in plan:
            g = self._stores[gi]
            have = len(g.pages[slot])
            new = g.pool.take(extra)
            g.pages[slot].extend(new)
            g.table_host[slot, have:have + extra] = torch.tensor(new, dtype=torch.int32)
            g.dirty = True

    def advance(self, slot: int, n: int) -> None:
        self._check_slot(slot)
        self.lengths[slot] += n

    def trim(self, slot: int) -> None:
        """Give back the pages ``slot`` holds beyond what its length needs (what a step
        reserved and then did not use because it failed)."""
        self._check_slot(slot)
        for g in self._stores:
            keep = g.pages_for(self.lengths[slot])
            extra = g.pages[slot][keep:]
            if extra:
                g.pool.give_back(extra)
                del g.pages[slot][keep:]

    def sync_tables(self) -> None:
        """Bring the device copies of changed page tables up to date."""
        for g in self._stores:
            if g.dirty:
                g.table.copy_(g.table_host, non_blocking=True)
                g.dirty = False

    def max_step_tokens(self, start: Optional[int] = None) -> int:
        """The most positions a step may add to a sequence (that holds ``start`` positions)."""
        return min([g.max_step_tokens(start) for g in self.groups] or [1 << 30])

    # ---- views --------------------------------------------------------
    def kv_view(self, entry: int) -> "KVView":
        gi, li = self._where[entry]
        g = self.groups[gi]
        c = g.cells
        if c is None:
            return KVView(g.k[li], g.v[li], g.table, g.page_tokens, g.ring_tokens, g.need,
                          fixed_tokens=g.fixed_tokens)
        return KVView(g.k[li], g.v[li], g.table, g.page_tokens, g.ring_tokens, g.need,
                      c.k[li], c.v[li], c.table, c.page_tokens)

    def has_kv(self, entry: int) -> bool:
        return entry in self._where

    def state_view(self, entry: int) -> torch.Tensor:
        return self.state[entry]

    def input_state_view(self, entry: int) -> torch.Tensor:
        return self.inputs[entry]

    def named_state(self, name: str) -> torch.Tensor:
        return self.named[name]

    def pages_in_use(self) -> int:
        return sum(g.n_pages - g.pool.n_free for g in self._stores)

    def bytes(self) -> int:
        return sum(g.bytes() for g in self.groups)


@dataclass
class KVView:
    """What a mixer sees of one schedule entry's keys and values."""

    k: torch.Tensor            # [pages, kv_heads, page_tokens, head_dim]
    v: torch.Tensor            # [pages, kv_heads, page_tokens, value_dim]
    page_table: torch.Tensor   # [slots, pages_per_seq] int32, on the device
    page_tokens: int
    ring_tokens: int           # 0: position p lives in cell p
    need: KVNeed
    # with ``need.pool``: the cells of the blocks, [pages, kv_heads, cell_page_tokens, width],
    # and their page table [slots, pages of cells per sequence]
    cell_k: Optional[torch.Tensor] = None
    cell_v: Optional[torch.Tensor] = None
    cell_table: Optional[torch.Tensor] = None
    cell_page_tokens: int = 0
    fixed_tokens: int = 0      # positions below it lie in cells of their own, ahead of the ring
