"""Attention backend of the paged engine: owns cache placement and masking for one ragged forward.

A decoder calls the backend once per layer run, ``backend(layer, q, k, v)`` for K/V attention,
``backend.latent(layer, mixer, q, c)`` for latent attention or ``backend.window(layer, mixer, q, k, v)`` for attention in a
window, with pooled blocks or differential; the backend writes the new rows into the pool at the step's slots and attends through the slot map.
``backend.recur(layer, mixer, *inputs)`` advances the recurrent states of the batch's sequences by what ``mixer.mix`` makes of
the inputs (or, for token trees, reads them and holds the nodes' inputs until a path is committed).
"""
from __future__ import annotations

from .. import ops


class PagedAttention:
    def __init__(self, pool, meta, scale: float = 1.0):
        self.pool, self.meta, self.scale = pool, meta, scale
        if pool.states is not None and not meta.causal:
            pool.states.begin_trees(meta.seq_rows.tolist(), meta.cu_q.tolist()[:-1])

    def __call__(self, layer, q, k, v):
        m = self.meta
        kp, vp = self.pool.layer(layer)
        ops.kv_scatter(k, v, kp, vp, m.slots)
        return ops.paged_tree_attention(q, kp, vp, self.pool.slot_map, m.seq_rows, m.cu_q, m.past_lens, m.mask_bits,
                                        self.scale, causal=m.causal, max_q=m.max_q)

    def latent(self, layer, mixer, q, c):
        m, pool = self.meta, self.pool.latent(layer)
        ops.latent_scatter(c, pool, m.slots)
        return ops.latent_attention(q, mixer.k_up.weight, mixer.v_up.weight, pool, self.pool.slot_map, m.seq_rows,
                                    m.cu_q, m.past_lens, m.mask_bits, mixer.cfg.scale, causal=m.causal, sink=mixer.sink)

    def window(self, layer, mixer, q, k, v):
        """``k`` is ``None`` where the layer uses another one's keys and values."""
        m, c = self.meta, mixer.cfg
        kp, vp = self.pool.layer(layer)
        blocks = self.pool.blocks(layer)
        if k is not None:
            ops.window_scatter(k, v, kp, vp, m.slots, maps=c.maps)
        if blocks is not None and m.causal:
            ops.pool_blocks(kp, vp, *blocks, self.pool.slot_map, m.seq_rows, m.cu_q, m.past_lens)
        return ops.window_attention(q, kp, vp, c.vdim, self.pool.slot_map, m.seq_rows, m.cu_q, m.past_lens, m.mask_bits, c.scale,
                                    c.window, mixer.sink, causal=m.causal, keep_first=c.keep_first, softcap=c.softcap, blocks=blocks,
                                    diff=mixer.differential())

    def recur(self, layer, mixer, *inputs):
        m, states = self.meta, self.pool.states
        if not m.causal:
            states.hold(layer, mixer, inputs)
        state, conv = states.layer(layer)
        return mixer.mix(inputs, state, conv, m.seq_rows, m.cu_q, m.past_lens, m.mask_bits, m.causal)

    delta = recur
