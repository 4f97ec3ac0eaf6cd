"""Recurrent state of the sequences a pool serves.

Per recurrent layer::

    state : (slots + 1, heads, dim, vdim)      fp32
    conv  : (slots + 1, taps, channels)        ring of the short convolutions' last inputs: position p in entry p % taps
                                               (None for a recurrence without convolutions)

A sequence's slot is its slot-map row in the paged pool.  Nothing is cleared when a slot changes hands: a forward whose
committed length is 0 starts from zeros whatever the slot holds.  The last slot belongs to no sequence; warm-up launches
of captured graphs write there.

A prompt portion or a decoded token advances the state in place.  A token tree does not, because most of its nodes are
rejected: the forward *holds* every node's inputs of the recurrence, and :meth:`commit` advances the state along the
accepted path from them.
"""
from __future__ import annotations

from typing import Callable, Optional

import torch


class StatePool:
    def __init__(self, shapes: list, slots: int, device="cpu", dtype=torch.float32):
        self.shapes, self.slots = list(shapes), int(slots)
        self.device = torch.device(device)
        self.state: list = []
        self.conv: list = []
        for c in self.shapes:
            self.state.append(None if c is None else torch.zeros(slots + 1, c.heads, c.dim, c.vdim, dtype=torch.float32, device=device))
            self.conv.append(None if c is None or not c.channels else torch.zeros(slots + 1, c.taps, c.channels, dtype=dtype, device=device))
        self._at: dict = {}          # state slot -> first row of its tree among the held rows
        self._advance = None
        self._held: dict = {}        # layer -> (mixer, recurrence inputs of every row of the last tree forward)

    @property
    def scratch(self) -> int:
        """The slot no sequence owns."""
        return self.slots

    def layer(self, i: int):
        return self.state[i], self.conv[i]

    def begin_trees(self, rows, starts, advance: Optional[Callable] = None) -> None:
        """A tree forward: the tree of state slot ``rows[j]`` occupies the batch's rows from ``starts[j]`` on.  A caller
        that holds the rows itself gives ``advance(row, past, start, path)``, which :meth:`commit` then calls."""
        self._at, self._held, self._advance = {int(r): int(s) for r, s in zip(rows, starts)}, {}, advance

    def hold(self, layer: int, mixer, inputs) -> None:
        """Keep a layer's recurrence inputs of a tree forward, the ones ``mixer.mix`` takes."""
        self._held[layer] = (mixer, inputs)

    def commit(self, row: int, past: int, path: torch.Tensor) -> None:
        """Advance slot ``row`` (at committed length ``past``) along the accepted nodes ``path`` of its held tree."""
        if row not in self._at:
            raise RuntimeError("no tree forward is held for this sequence")
        start, n = self._at.pop(row), int(path.numel())
        if n == 0:
            return
        if self._advance is not None:
            return self._advance(row, past, start, path.to(self.device))
        idx = path.to(self.device).long() + start
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=self.device)
        rows, cu_q, past_t = i32([row]), i32([0, n]), i32([past])
        for i, (mixer, inputs) in self._held.items():
            mixer.mix([x[idx] for x in inputs], self.state[i], self.conv[i], rows, cu_q, past_t, None, True)
