"""Fused kernel form of a pre-norm decoder whose layers hold attention over K/V heads, latent attention or retention in any
order (Kizezen, Sogidra) for the engine's kernel path.

Per layer, on ``h``, the bf16 norm of the fp32 residual stream ``x``:

1. ONE input GEMM: what stays 32-bit behind it (gate logits, the latent row) leaves as fp32, every other projection as bf16;
2. the mixer (:mod:`~jetspec_b200.engine.mixers`): one kernel behind the projections and the attention with sinks and gates
   folded in, or the retention kernels;
3. the output GEMM adds to the stream, one kernel norms it;
4. feed-forward: up GEMM with the activation (exact gelu, xIELU) in its epilogue, down GEMM that adds to the stream, the next
   norm (behind the last layer the model's final one).

Where sublayers have a norm on their output too, the output GEMM leaves bf16 rows and ONE kernel norms them, adds them to the
stream and norms the sum; at a layer's end it also keeps the layer's result and makes the weighted sum over the depth.

The embedding kernel adds learned positions, norms its rows for the first layer and makes the (cos, sin) tables of all layers'
rotations.

Token trees leave the recurrent states alone and keep every retention layer's projections, and pool no blocks;
:meth:`PreNormStack.commit` then advances the states along the accepted nodes and pools the blocks they complete.
"""
from __future__ import annotations

import types

import torch

from ..models.config import LatentAttentionConfig, WindowAttentionConfig
from ..models.layers import XieluMLP
from ..ops import cuda_ext as X
from .latent_stack import latent_part, latent_parts
from .mixers import LatentMixer, RetentionMixer, WindowMixer, pad, pad_heads, up


class _LayerWeights:
    """Kernel-ready weights of one layer."""

    def __init__(self, layer, cfg, i: int, wp: int):
        mix, c, W, eps = layer.mixer, cfg.layers[i].mixer, cfg.hidden_size, cfg.norm_eps
        f32 = lambda p: p.detach().float().contiguous()
        self.index, self.eps, self.rot_at = i, eps, 0
        self.kind, raw = cfg.layers[i].mixer_type, []
        row = lambda n: pad(n.scale().detach().view(1, -1), 1, wp).view(-1)
        if isinstance(c, WindowAttentionConfig):
            self.kind = "attention"
            self.mix = WindowMixer(mix, eps, wp)
            act = torch.cat(self.mix.qkv, 0)                   # read as unpadded rows
            raw = [self.mix.gate] if c.gate else []
            self.gate_at, self.w_o = 0, self.mix.w_o
        elif isinstance(c, LatentAttentionConfig):
            self.mix = LatentMixer(mix)
            act = pad_heads(mix.q_proj.weight.detach(), c.heads, self.mix.dp, W)
            raw = [mix.kv_down.weight.detach()] + ([mix.gate_proj.weight.detach()] if c.gate else [])
            self.gate_at, self.w_o = c.row, pad(self.mix.w_o, wp, up(self.mix.out_cols, 8))
            self.kv_norm = f32(mix.kv_norm)
        else:
            self.mix = RetentionMixer(mix, eps, wp)
            act = torch.zeros(self.mix.act_cols, W, dtype=mix.q_proj.weight.dtype, device=mix.q_proj.weight.device)
            for o, w in zip(self.mix.offs, self.mix.weights):
                act[o:o + w.shape[0]] = w
            self.w_o = self.mix.w_o
        self.gated = bool(getattr(c, "gate", False))
        self.n_raw = up(sum(w.shape[0] for w in raw), 128) if raw else 0
        self.act_cols = up(act.shape[0], 128)
        blocks = [pad(torch.cat(raw, 0), self.n_raw, wp)] if raw else []
        self.w_in = torch.cat(blocks + [pad(act, self.act_cols, wp)], 0)
        self.norm1, self.ff = row(layer.norm1), 0
        self.out1 = row(layer.norm1b) if hasattr(layer, "norm1b") else None      # norms on the sublayers' outputs
        self.depth = f32(layer.dwa) if hasattr(layer, "dwa") else None
        if layer.mlp is not None:
            self.ff = up(layer.mlp.up_proj.weight.shape[0], 128)
            self.w_up = pad(layer.mlp.up_proj.weight.detach(), self.ff, wp)
            self.w_down = pad(layer.mlp.down_proj.weight.detach(), wp, self.ff)
            self.norm2 = row(layer.norm2)
            self.out2 = row(layer.norm2b) if self.out1 is not None else None
            self.act = dict(act=X.ACT_XIELU, act_args=layer.mlp.coefficients()) if isinstance(layer.mlp, XieluMLP) else dict(act=X.ACT_GELU_ERF)


class PreNormStack:
    """Weights of the whole decoder, prepared once, and the launch sequence over them."""

    def __init__(self, model, device):
        cfg = model.config
        self.cfg, self.device = cfg, torch.device(device)
        self.width, self.wp = cfg.hidden_size, up(cfg.hidden_size, 8)
        self.layers = [_LayerWeights(l, cfg, i, self.wp) for i, l in enumerate(model.model.layers)]
        self.final_norm = pad(model.model.norm.scale().detach().view(1, -1), 1, self.wp).view(-1)
        table, head = model.model.embed_tokens.weight.detach(), model.lm_head.weight.detach()
        self.table, self.head = (w if self.wp == self.width else pad(w, w.shape[0], self.wp) for w in (table, head))
        pos = getattr(model.model, "pos_embed", None)
        self.pos_table = pad(pos.weight.detach(), pos.weight.shape[0], self.wp) if pos is not None else None
        self.vocab, self.embed_scale = cfg.vocab_size, float(cfg.embed_scale)
        self.depth = self.layers[0].depth is not None
        self.pooled = [L for L in self.layers if getattr(L.mix.cfg, "pool", 0)]
        self._rotations()
        self.recurrent = [L for L in self.layers if L.kind == "retention"]
        self.may_expand = any(L.kind == "latent_attention" and L.mix.expand for L in self.layers)

    def _rotations(self) -> None:
        """Frequencies and amplitudes of all layers' rotations side by side; equal rotations share their columns, and every
        rotation starts at an even one (vector loads)."""
        at, freq, amp = {}, [], []
        for L in self.layers:
            r = L.mix.cfg.rot
            if r is None:
                continue
            key = (r.dims, r.base, r.scaling)              # the pairing does not enter the table
            if key not in at:
                at[key] = len(freq)
                f = r.frequencies()
                extra = len(f) % 2
                freq += f + [0.0] * extra
                amp += [r.amplitude()] * (len(f) + extra)
            L.rot_at = at[key]
        self.n_freq = max(2, len(freq))
        t = lambda v: torch.tensor(v + [0.0] * (self.n_freq - len(v)), dtype=torch.float32, device=self.device)
        self.freq, self.amp = t(freq), t(amp)

    @staticmethod
    def caches(pool):
        """What :meth:`run` needs of a pool."""
        return pool

    # ------------------------------------------------------------------ buffers
    def buffers(self, T: int, max_keys: int) -> "types.SimpleNamespace":
        """Activation buffers for ``T`` rows; ``max_keys`` bounds a sequence's cache length (key splits)."""
        dev, cols = self.device, {}
        b = types.SimpleNamespace(T=T, max_keys=max_keys, cols=cols, ws={})
        b.x = torch.zeros(T, self.wp, dtype=torch.float32, device=dev)
        b.h = torch.zeros(T, self.wp, dtype=torch.bfloat16, device=dev)
        # embedding output and every layer's result
        b.hist = torch.empty(len(self.layers) + 1, T, self.wp, dtype=torch.float32, device=dev) if self.depth else None
        b.rot = torch.zeros(T, self.n_freq, 2, dtype=torch.float32, device=dev)

        def get(name, c, dtype=torch.bfloat16, rows=T, zero=False):
            key = (name, c, rows)
            if key not in cols:
                cols[key] = (torch.zeros if zero else torch.empty)(rows, c, dtype=dtype, device=dev)
            return cols[key]
        b.get = get
        return b

    def _act(self, st, L, hold: bool) -> torch.Tensor:
        """A layer's bf16 projections; a retention layer's outlive the forward of a token tree."""
        return st.get(f"act{L.index}" if hold and L.kind == "retention" else "act", L.act_cols)

    def _rot(self, st, L) -> torch.Tensor:
        return st.rot[:, L.rot_at:]

    # ------------------------------------------------------------------ one forward
    def run(self, st, ids, pool, batch, xn, taps=None, tap_ids=None, pdl: bool = True) -> int:
        """Embed ``ids (T,)`` int32 and run every layer on ``st``; ``xn (T, wp)`` gets the final norm's output.  Returns
        the number of kernels launched."""
        lib, p = X.load(), X._p
        T, n, last = st.T, 1, len(self.layers) - 1
        X._check(lib.js_embed_rms(p(ids), p(self.table), self.vocab, self.table.stride(0), X.ctypes.c_float(self.embed_scale),
                                  p(self.layers[0].norm1), X.ctypes.c_float(self.layers[0].eps), p(st.x if not self.depth else st.hist[0]), p(st.h),
                                  self.wp, T, self.width, p(batch.positions), p(self.pos_table),
                                  self.pos_table.shape[0] if self.pos_table is not None else 0, p(self.freq), p(self.amp), self.n_freq, p(st.rot), int(pdl), X._stream()),
                 "js_embed_rms")
        tap_ids = list(tap_ids) if taps is not None else []
        for i, L in enumerate(self.layers):
            tap = None
            if i in tap_ids and i != last:
                j = tap_ids.index(i)
                tap = taps[:, j * self.width:(j + 1) * self.width]
            norm, h = (self.layers[i + 1].norm1, st.h) if i != last else (self.final_norm, xn)
            n += self._layer(st, L, pool, batch, norm, h, tap, pdl)
        for j, t in enumerate(tap_ids):
            if t == last:
                taps[:, j * self.width:(j + 1) * self.width].copy_(xn[:, : self.width])
            elif tap_ids.index(t) != j:
                k = tap_ids.index(t)
                taps[:, j * self.width:(j + 1) * self.width].copy_(taps[:, k * self.width:(k + 1) * self.width])
        return n

    def _norm(self, st, w, eps, h, tap, pdl) -> None:
        p = X._p
        assert h.stride(0) == st.x.stride(0)
        X._check(X.load().js_rms_rows(p(st.x), p(w), X.ctypes.c_float(eps), p(h), self.wp, st.T, self.width, p(tap),
                                      tap.stride(0) if tap is not None else 0, int(pdl), X._stream()), "js_rms_rows")

    def _layer(self, st, L, pool, batch, norm, h, tap, pdl) -> int:
        """One layer on ``st.h``; the norm behind it (weights ``norm``) goes to ``h``."""
        raw = st.get("raw", L.n_raw, torch.float32) if L.n_raw else None
        act = self._act(st, L, batch.mask is not None)
        X.gemm_inproj(st.h, L.w_in, raw, L.n_raw, act, False, pdl=pdl, act=X.ACT_NONE)
        gate = raw[:, L.gate_at:] if L.gated else None
        rot = self._rot(st, L)
        if L.kind == "attention":
            o, n = L.mix.run(st, pool.layer(L.index), batch, act, gate, rot, pdl, pdl, blocks=pool.blocks(L.index))
        elif L.kind == "latent_attention":
            o, n = self._latent(st, L, pool.latent(L.index), batch, raw, act, gate, rot, pdl)
        else:
            o, n = L.mix.run(st, pool.states.layer(L.index)[0], batch, act, rot, pdl)
        if L.out1 is not None:
            return n + self._normed(st, L, o, norm, h, tap, pdl)
        X.gemm_resid32(o, L.w_o, st.x, pdl=pdl)
        n += 3
        if not L.ff:
            self._norm(st, norm, L.eps, h, tap, pdl)
            return n
        self._norm(st, L.norm2, L.eps, st.h, None, pdl)
        a = st.get("ff", L.ff)
        X.gemm_inproj(st.h, L.w_up, None, 0, a, False, pdl=pdl, **L.act)
        X.gemm_resid32(a, L.w_down, st.x, pdl=pdl)
        self._norm(st, norm, L.eps, h, tap, pdl)
        return n + 3

    def _normed(self, st, L, o, norm, h, tap, pdl) -> int:
        """What follows the mixer where sublayers have norms on their outputs.  Returns the launches, the input GEMM's included."""
        y = st.get("y", self.wp)
        X.gemm(o, L.w_o, out=y, pdl=pdl)
        x = st.hist[0] if self.depth and L.index == 0 else st.x        # the embedding output stays as it is
        end = dict(hist=st.hist, d=L.depth, tap=tap, pdl=pdl)
        if not L.ff:
            X.sandwich(y, x, L.out1, st.x, norm, L.eps, h, self.width, **end)
            return 3
        X.sandwich(y, x, L.out1, st.x, L.norm2, L.eps, st.h, self.width, pdl=pdl)
        a = st.get("ff", L.ff)
        X.gemm_inproj(st.h, L.w_up, None, 0, a, False, pdl=pdl, **L.act)
        X.gemm(a, L.w_down, out=y, pdl=pdl)
        X.sandwich(y, st.x, L.out2, st.x, norm, L.eps, h, self.width, **end)
        return 6

    def _latent(self, st, L, pool, batch, raw, act, gate, rot, pdl):
        m, c, p = L.mix, L.mix.cfg, X._p
        q = act[:, : c.heads * m.dp]
        X._check(X.load().js_latent_rot_post(
            p(raw), raw.stride(0), c.kv_rank, c.rot_dim, p(L.kv_norm), X.ctypes.c_float(L.eps), p(pool), m.rp, pool.shape[0], p(batch.slots),
            p(q), q.stride(0), c.heads, m.dp, c.dim, p(rot), rot.stride(0) // 2, st.T, p(X.status_word(self.device)), int(pdl), X._stream()),
            "js_latent_rot_post")
        o = st.get("lo", up(m.out_cols, 8), zero=True)
        return o, 1 + m.attend(st, pool, batch, q, o, gate, pdl)

    # ------------------------------------------------------------------ token trees
    def commit(self, st, pool, state_rows, cu_q, past, path, path_len, pdl: bool = True) -> int:
        """Advance one sequence's states along the rows ``path[:path_len]`` (device) of the tree forward run on ``st`` and pool the
        blocks they complete; ``past`` is the committed length behind the path."""
        for L in self.pooled:
            X.pool_blocks(*pool.layer(L.index), *pool.blocks(L.index), pool.slot_map, state_rows, None, past, counts=path_len,
                          most=path.numel(), pdl=pdl)
        for L in self.recurrent:
            L.mix.advance(self._act(st, L, True), self._rot(st, L), pool.states.layer(L.index)[0], state_rows, cu_q, past, path, path_len, pdl)
        return len(self.recurrent) + len(self.pooled)

    def hold_trees(self, st, pool, rows, starts, nodes: int) -> None:
        """Register the tree forward on ``st`` with the state pool: the tree of state slot ``rows[j]`` begins at row
        ``starts[j]`` and has up to ``nodes`` rows."""
        i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=self.device)

        def advance(row, past, start, path):
            end = min(start + nodes, st.T)
            self.commit(st, pool, i32([row]), i32([start, end]), i32([past + path.numel()]), path.to(torch.int32), i32([path.numel()]))
        pool.states.begin_trees(rows, starts, advance)

    # ------------------------------------------------------------------ batches
    def uniform_batch(self, slot_map, seq_rows, cu_q, past, slots, mask, causal, rows, max_q, max_keys, positions=None, state_rows=None):
        """A batch of equal row counts (decode steps and token trees); one row a sequence is a plain decode step."""
        return types.SimpleNamespace(slot_map=slot_map, seq_rows=seq_rows, cu_q=cu_q, past=past, slots=slots,
                                     mask=None if causal or max_q == 1 else mask, positions=positions, max_keys=max_keys, max_rows=max_q,
                                     state_rows=seq_rows if state_rows is None else state_rows,
                                     parts=[latent_part(0, rows, seq_rows, cu_q, past, max_q, max_keys)])

    def ragged_batch(self, slot_map, meta, counts, past_lens):
        """Portions of prompts beside decoded tokens, or token trees."""
        return types.SimpleNamespace(slot_map=slot_map, seq_rows=meta.seq_rows, cu_q=meta.cu_q, past=meta.past_lens, slots=meta.slots,
                                     mask=None if meta.causal else meta.mask_bits, positions=meta.positions,
                                     max_keys=max(a + b for a, b in zip(counts, past_lens)), max_rows=max(counts), state_rows=meta.seq_rows,
                                     parts=latent_parts(slot_map, meta, counts, past_lens, self.may_expand))
