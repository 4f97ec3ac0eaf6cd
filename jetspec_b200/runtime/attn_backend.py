"""Attention backend of the paged engine: owns cache placement and masking for one ragged forward.

A decoder calls the backend once per layer run, ``backend(layer, q, k, v)`` for K/V attention or
``backend.latent(layer, mixer, q, c)`` for latent attention; the backend writes the new rows into the pool at the
step's slots and attends through the slot map.
"""
from __future__ import annotations

from .. import ops


class PagedAttention:
    def __init__(self, pool, meta, scale: float = 1.0):
        self.pool, self.meta, self.scale = pool, meta, scale

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
                                    m.cu_q, m.past_lens, m.mask_bits, mixer.cfg.scale, causal=m.causal)
