"""Slot-addressed paged KV pool.

One pool serves every layer and every sequence::

    k_pool, v_pool : (L, Hkv, S, D)       S = num_pages * page_size slots
    slot_map       : (max_seqs, max_len)  int32, on the device

A model whose attention caches one latent row per token instead of K and V heads gets, per cache layer, a pool of
rows of that layer's own width (rounded up to 64 elements, the rest stays zero)::

    latent_pools : list of (S, width)

A model whose layers differ gets its K and V pools per layer, ``(Hkv, S, width)`` (or nothing where a layer caches
nothing), and one with recurrent layers also a :class:`~jetspec_b200.runtime.state_pool.StatePool`: a sequence's state
slot is its slot-map row, so it is granted, given back, evicted and used again together with the row::

    kv_layers : list of (k_pool, v_pool) or None
    states    : StatePool or None

Kinds can differ from layer to layer: ``kv_layers`` and ``latent_pools`` then hold ``None`` where a layer caches the other kind
or nothing.  A layer that uses another layer's keys and values has that layer's pools in ``kv_layers``.

A layer whose attention sees whole blocks of ``P`` tokens through one pooled key and value keeps these beside its K and V::

    kv_blocks  : list of (k_pool, v_pool) or None    (Hkv, num_pages * ceil(page_size / P), width)
    block_maps : {P: (max_seqs, max_len // P)}       row of every block of a sequence

A block's row belongs to the logical page its last token lies in, so blocks are granted, given back and used again with the
pages.  Tokens may trade slots inside a sequence (below); blocks never do.  A block is pooled when its last token is
committed: in the forward of a prompt portion or decoded token, or when a path of a token tree is committed
(:meth:`PagedKVPool.pool_committed`).

Everything below the buffers (pages, slot maps, admission, eviction, commit) is the same for all kinds.

A *page* (``page_size`` consecutive slots) is the unit of allocation and is shared
by all layers (one page id addresses the same slots in each layer's slice), so a
sequence of ``n`` tokens owns ``ceil(n / page_size)`` ids, not ``L`` times that.
A *slot map row* translates a sequence's logical position to a slot.  Attention
reads K/V through the slot map, so committing an accepted tree path never moves
KV bytes: it only permutes the ``N`` slot-map entries of the tree window so that
the accepted nodes' slots come first (positions ``past .. past+k``) and the
rejected nodes' slots are recycled for the next round's tree.  Memory in use is
therefore exactly ``committed tokens + tree window``, with nothing leaked between
rounds.

Compared with the reference cache (``jetspec/inference_engine/paged_kv_cache.py``):
same responsibilities (admission, allocation, eviction with LRU, refcounts, status,
``EvictionRequired`` / ``EvictionFailed``), but layer-shared page ids from the start
(the reference allocates distinct ids per layer, ``:189-203``), O(1) free-list
operations, and no per-step host-side block-table rebuild (``:867-883``).
"""
from __future__ import annotations

import itertools
from collections import deque
from dataclasses import dataclass, field
from typing import Optional

import torch

from .state_pool import StatePool


class EvictionRequired(RuntimeError):
    """The pool cannot serve the request without evicting another sequence."""


class EvictionFailed(RuntimeError):
    """No sequence can be evicted (nothing else is resident)."""


def latent_row_width(width: int) -> int:
    """Elements a cached latent row takes: ``width`` rounded up to 64 (one 128-byte line of bf16)."""
    return (int(width) + 63) // 64 * 64


def window_row_width(dim: int, vdim: int, dtype: torch.dtype, maps: int = 1) -> tuple:
    """Elements a K and a V row take: bf16 heads of up to 128 are padded to the tensor-core attention's 128.  The keys of a
    head's ``maps`` lie side by side in its row, an equal share of it each."""
    return (128, 128) if dtype == torch.bfloat16 and max(dim * maps, vdim) <= 128 else (int(dim) * maps, int(vdim))


@dataclass
class SeqState:
    seq_id: int
    row: int
    pages: list = field(default_factory=list)
    length: int = 0          # committed KV length (logical positions with valid KV)
    capacity: int = 0        # slots granted (positions that have a slot id in the map)
    last_used: int = 0


class PagedKVPool:
    def __init__(self, num_layers: int, num_kv_heads: int, head_dim: int, num_pages: int,
                 page_size: int = 16, max_seqs: int = 64, max_seq_len: int = 4096,
                 device="cpu", dtype=torch.float32, latent_widths: Optional[list] = None,
                 kv_shapes: Optional[list] = None, state_shapes: Optional[list] = None,
                 kv_sources: Optional[list] = None, kv_pools: Optional[list] = None):
        self.num_layers, self.num_kv_heads, self.head_dim = num_layers, num_kv_heads, head_dim
        self.page_size, self.num_pages = int(page_size), int(num_pages)
        self.max_seqs, self.max_seq_len = int(max_seqs), int(max_seq_len)
        self.device, self.dtype = torch.device(device), dtype
        S = self.num_pages * self.page_size
        self.k_pool = self.v_pool = self.latent_pools = self.kv_layers = self.states = self.kv_blocks = None
        self.block_maps: dict = {}
        if kv_shapes is not None:
            def pools(rows, heads, dim, vdim, maps=1):
                return tuple(torch.zeros(heads, rows, w, dtype=dtype, device=device) for w in window_row_width(dim, vdim, dtype, maps))
            self.kv_layers = [pools(S, *shape) if shape is not None else None for shape in kv_shapes]
            if kv_sources is not None:
                self.kv_layers = [self.kv_layers[j] for j in kv_sources]
            if kv_pools is not None and any(kv_pools):
                self.block_sizes = list(kv_pools)
                self.kv_blocks = [pools(self.num_pages * self._blocks_per_page(P), *shape) if P else None for P, shape in zip(kv_pools, kv_shapes)]
                self.block_maps = {P: torch.zeros(self.max_seqs, max(1, self.max_seq_len // P), dtype=torch.int32, device=device)
                                   for P in set(kv_pools) if P}
        if latent_widths is not None:
            self.latent_pools = [None if w is None else torch.zeros(S, latent_row_width(w), dtype=dtype, device=device)
                                 for w in latent_widths]
        if kv_shapes is None and latent_widths is None:
            self.k_pool = torch.zeros(num_layers, num_kv_heads, S, head_dim, dtype=dtype, device=device)
            self.v_pool = torch.zeros(num_layers, num_kv_heads, S, head_dim, dtype=dtype, device=device)
        if state_shapes is not None:
            self.states = StatePool(state_shapes, self.max_seqs, device=device, dtype=dtype)
        self.slot_map = torch.zeros(self.max_seqs, self.max_seq_len, dtype=torch.int32, device=device)
        self._free_pages: deque = deque(range(self.num_pages))
        self._refcount = [0] * self.num_pages
        self._free_rows: deque = deque(range(self.max_seqs))
        self._seqs: dict = {}
        self._clock = itertools.count(1)
        self.frozen = False   # set while CUDA graphs hold pointers into the pool

    # -- sizing ---------------------------------------------------------------
    @classmethod
    def for_model(cls, cfg, num_pages: int, world: int = 1, **kw) -> "PagedKVPool":
        """A pool of the shape ``cfg``'s attention caches (``world``: ranks the K/V heads are sharded over)."""
        widths, shapes = cfg.latent_widths(), cfg.kv_shapes()
        if widths is not None or shapes is not None:
            optional = {k: getattr(cfg, k)() for k in ("kv_sources", "kv_pools") if hasattr(cfg, k)}
            return cls(cfg.num_hidden_layers, 0, 0, num_pages, latent_widths=widths, kv_shapes=shapes, state_shapes=cfg.state_shapes(),
                       **optional, **kw)
        return cls(cfg.num_hidden_layers, cfg.num_key_value_heads // world, cfg.head_dim, num_pages, **kw)

    @property
    def num_slots(self) -> int:
        return self.num_pages * self.page_size

    def pages_for(self, tokens: int) -> int:
        return (int(tokens) + self.page_size - 1) // self.page_size

    @property
    def free_page_count(self) -> int:
        return len(self._free_pages)

    def utilization(self) -> float:
        return 1.0 - len(self._free_pages) / max(1, self.num_pages)

    def layer(self, li: int):
        return self.kv_layers[li] if self.kv_layers is not None else (self.k_pool[li], self.v_pool[li])

    def latent(self, li: int) -> torch.Tensor:
        return self.latent_pools[li]

    def _blocks_per_page(self, P: int) -> int:
        """Most blocks of ``P`` tokens that end in one page."""
        return (self.page_size + P - 1) // P

    def blocks(self, li: int):
        """``(k rows, v rows, block map, P)`` of a layer's pooled blocks, or ``None``."""
        if self.kv_blocks is None or self.kv_blocks[li] is None:
            return None
        P = self.block_sizes[li]
        return (*self.kv_blocks[li], self.block_maps[P], P)

    def _map_blocks(self, st: "SeqState", base: int) -> None:
        """Rows of the blocks that end at position ``base`` or later in the pages of ``st``."""
        for P, table in self.block_maps.items():
            first, stop = base // P, min(len(st.pages) * self.page_size // P, table.shape[1])
            if stop > first:
                b = torch.arange(first, stop)
                page = ((b + 1) * P - 1) // self.page_size
                rows = torch.tensor(st.pages)[page] * self._blocks_per_page(P) + b - page * self.page_size // P
                table[st.row, first:stop] = rows.to(torch.int32).to(self.device, non_blocking=True)

    def pool_committed(self, row: int, past: int, n: int) -> None:
        """Pool the blocks whose last token is among the positions ``[past, past + n)`` of slot-map row ``row``."""
        if self.kv_blocks is None or n <= 0:
            return
        done = [li for li, P in enumerate(self.block_sizes) if P and (past + n) // P > past // P]
        if not done:
            return
        from .. import ops
        i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=self.device)
        rows, cu_q, past_t = i32(row), i32(0, n), i32(past)
        for li in done:
            ops.pool_blocks(*self.kv_layers[li], *self.blocks(li), self.slot_map, rows, cu_q, past_t)

    # -- sequences ------------------------------------------------------------
    def has(self, seq_id: int) -> bool:
        return seq_id in self._seqs

    def state(self, seq_id: int) -> SeqState:
        return self._seqs[seq_id]

    def touch(self, seq_id: int) -> None:
        self._seqs[seq_id].last_used = next(self._clock)

    def reclaimable_pages(self, exclude: Optional[int] = None) -> int:
        return sum(len(s.pages) for sid, s in self._seqs.items() if sid != exclude)

    def admit_sequence(self, seq_id: int, num_tokens: int) -> bool:
        """True when ``num_tokens`` positions could be granted, counting pages that
        evicting *other* sequences would free."""
        if num_tokens > self.max_seq_len:
            return False
        have = len(self._seqs[seq_id].pages) if seq_id in self._seqs else 0
        need = self.pages_for(num_tokens) - have
        if seq_id not in self._seqs and not self._free_rows and not self._seqs:
            return False
        return need <= len(self._free_pages) + self.reclaimable_pages(exclude=seq_id)

    def allocate_slots(self, seq_id: int, num_tokens: int, allow_evict: bool = True) -> bool:
        """Grant slots so that positions ``[0, num_tokens)`` are mapped; evicts least-recently
        used *other* sequences if the free list is short.  False when it cannot fit."""
        if num_tokens > self.max_seq_len:
            return False
        st = self._seqs.get(seq_id)
        if st is None:
            if not self._free_rows:
                if not allow_evict:
                    return False
                try:
                    self.evict_sequence(exclude=seq_id)
                except EvictionFailed:
                    return False
            st = SeqState(seq_id, self._free_rows.popleft(), last_used=next(self._clock))
            self._seqs[seq_id] = st
        need = self.pages_for(num_tokens) - len(st.pages)
        while need > len(self._free_pages):
            if not allow_evict:
                return False
            try:
                self.evict_sequence(exclude=seq_id)
            except EvictionFailed:
                return False
        if need > 0:
            new_pages = [self._free_pages.popleft() for _ in range(need)]
            for p in new_pages:
                assert self._refcount[p] == 0, f"page {p} handed out twice"
                self._refcount[p] = 1
            base = len(st.pages) * self.page_size
            st.pages.extend(new_pages)
            ids = (torch.tensor(new_pages, dtype=torch.int32).repeat_interleave(self.page_size) * self.page_size
                   + torch.arange(self.page_size, dtype=torch.int32).repeat(len(new_pages)))
            end = min(base + ids.numel(), self.max_seq_len)
            self.slot_map[st.row, base:end] = ids[: end - base].to(self.device, non_blocking=True)
            if self.block_maps:
                self._map_blocks(st, base)
        st.capacity = min(len(st.pages) * self.page_size, self.max_seq_len)
        st.last_used = next(self._clock)
        return True

    def reserve(self, seq_id: int, num_tokens: int) -> None:
        """Like :meth:`allocate_slots` but never evicts and raises when it does not fit."""
        if not self.allocate_slots(seq_id, num_tokens, allow_evict=False):
            raise EvictionRequired(f"sequence {seq_id} needs {self.pages_for(num_tokens)} pages; "
                                   f"{len(self._free_pages)} free")

    def free(self, seq_id: int) -> None:
        st = self._seqs.pop(seq_id, None)
        if st is None:
            return
        for p in st.pages:
            self._refcount[p] -= 1
            assert self._refcount[p] >= 0, f"page {p} refcount went negative"
            if self._refcount[p] == 0:
                self._free_pages.append(p)
        self._free_rows.append(st.row)

    def evict_sequence(self, seq_id: Optional[int] = None, exclude: Optional[int] = None) -> int:
        """Drop a resident sequence (named, or the least recently used one) and return its id."""
        if seq_id is None:
            cands = [s for sid, s in self._seqs.items() if sid != exclude]
            if not cands:
                raise EvictionFailed("no evictable sequence resident")
            seq_id = min(cands, key=lambda s: s.last_used).seq_id
        elif seq_id not in self._seqs:
            raise EvictionFailed(f"sequence {seq_id} is not resident")
        self.free(seq_id)
        return seq_id

    def crop(self, seq_id: int, length: int) -> None:
        st = self._seqs[seq_id]
        if self.states is not None and 0 < int(length) < st.length:
            raise RuntimeError("a recurrent state cannot be cropped to an earlier position")
        st.length = min(st.length, int(length))

    def reset(self) -> None:
        for sid in list(self._seqs):
            self.free(sid)

    def resident(self) -> list:
        return list(self._seqs)

    def get_seq_status(self, seq_id: int) -> dict:
        st = self._seqs[seq_id]
        return {"seq_id": seq_id, "row": st.row, "length": st.length, "capacity": st.capacity,
                "pages": len(st.pages), "last_used": st.last_used}

    # -- tree window ------------------------------------------------------------
    def commit_path(self, seq_id: int, past: int, num_nodes: int, path) -> None:
        """Make the accepted nodes' slots the next committed positions.

        ``path`` lists accepted node indices (root first).  The window
        ``slot_map[row, past:past+num_nodes]`` is permuted to ``path`` followed by the
        remaining nodes in index order, and the committed length becomes
        ``past + len(path)``.  No KV bytes move; recurrent states advance along the path, and
        blocks it completes are pooled.
        """
        st = self._seqs[seq_id]
        if isinstance(path, (list, tuple)):      # host path: the permutation is built without a device read
            taken = set(path)
            order = torch.tensor(list(path) + [i for i in range(num_nodes) if i not in taken], dtype=torch.long,
                                 device=self.device)
            n_path = len(path)
        else:
            p = torch.as_tensor(path, dtype=torch.long, device=self.device)
            keep = torch.ones(num_nodes, dtype=torch.bool, device=self.device)
            keep[p] = False
            order = torch.cat((p, torch.nonzero(keep, as_tuple=True)[0]))
            n_path = int(p.numel())
        if self.states is not None:
            self.states.commit(st.row, past, order[:n_path])
        win = self.slot_map[st.row, past:past + num_nodes]
        self.slot_map[st.row, past:past + num_nodes] = win[order]
        self.pool_committed(st.row, past, n_path)
        st.length = past + n_path
        st.last_used = next(self._clock)
