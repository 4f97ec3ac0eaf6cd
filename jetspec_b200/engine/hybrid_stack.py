"""Fused kernel form of a decoder of window attention, gated delta rules and table-routed experts (Zasipel) for the
engine's kernel path.

Per layer, on the bf16 copy ``h`` of the fp32 residual stream ``x``:

1. ONE input GEMM: step-size and decay logits leave as fp32, every other projection of the layer (both mixers' q, k, v
   and the output gate, or its low-rank factors) as bf16; a channel-decay layer's second low-rank factors are one more
   GEMM over both factors side by side;
2. window attention: one kernel adds the biases, rotates and norms q and k and scatters K/V to the pool; the tcgen05
   attention kernel follows, with its key range cut to the window and the sink in its softmax;
3. delta rule: a decode step is one kernel from the projections to the gated per-head norm; portions go in blocks of 8
   rows (one kernel prepares all blocks, one walks them, the norm follows); token trees go row by row;
4. output GEMMs, then ONE kernel for the residual step: the norms of the sublayers' outputs, the sum, the stream, the
   next bf16 input (and behind the last layer the model's final norm);
5. experts: the permutation by expert depends on the token ids alone, so one launch at the start makes every layer's;
   two grouped GEMMs, the shared expert's two GEMMs, and the same residual kernel as the combine.

Two branches of a layer do not depend on each other: window attention and delta rule, shared expert and routed experts.
In captured graphs and on long portions they run on two streams: each alone leaves most of the device idle.

Token trees leave the recurrent states alone and keep every layer's prepared rows; :meth:`HybridStack.commit` then
advances the states along the accepted nodes.  Every size is padded to what the kernels want when the weights are
prepared; padding is zero and stays zero.
"""
from __future__ import annotations

import types

import numpy as np
import torch

from ..ops import cuda_ext as X
from .latent_stack import MAX_SORT_PAIRS
from .mixers import WindowMixer, pad, up

FORK_MIN_TOKENS = 512          # eager launches fork from this many rows on (below, the host is what a forward waits for)

_TABLE_LAYER = np.dtype([("table", "<u8"), ("top", "<i4"), ("experts", "<i4"), ("off", "<i4"), ("pad", "<i4")])


def _cols(parts, align: int = 8):
    """Offsets of consecutive column blocks, each starting on a multiple of ``align``, and the end."""
    offs, at = [], 0
    for n in parts:
        offs.append(at)
        at = up(at + n, align)
    return offs, at


def _stack_rows(ws, offs, rows: int, cols: int) -> torch.Tensor:
    """Weights ``ws`` as row blocks at ``offs`` of a zero ``(rows, cols)`` matrix."""
    out = torch.zeros(rows, cols, dtype=ws[0].dtype, device=ws[0].device)
    for w, o in zip(ws, offs):
        out[o:o + w.shape[0], : w.shape[1]] = w
    return out


def _interleave(gate: torch.Tensor, up: torch.Tensor, ff: int, cols: int) -> torch.Tensor:
    return X.interleave_gate_up(pad(gate, ff, cols), pad(up, ff, cols), 128)


class _LayerWeights:
    """Kernel-ready weights of one layer."""

    def __init__(self, layer, cfg, i: int, wp: int):
        l, W = cfg.layers[i], cfg.hidden_size
        f32 = lambda p: p.detach().float().contiguous()
        d, self.dc = layer.delta, l.delta
        c = self.dc
        self.index, self.parallel = i, l.window is not None
        ws, names = [], []

        def add(name, w):
            names.append(name)
            ws.append(w.detach())

        if self.parallel:
            self.win = WindowMixer(layer.mixer.left, cfg.norm_eps, wp)
            for n, w in zip("qkv", self.win.qkv):
                add("w" + n, w)
            self.left_norm, self.right_norm = f32(layer.mixer.left_norm.weight), f32(layer.mixer.right_norm.weight)
        raw = [d.beta_proj.weight.detach()]
        if not c.decay_rank:
            raw.append(d.decay_proj.weight.detach())
        for n in "qkv":
            add(n, getattr(d, n + "_proj").weight)
        low = []
        if c.decay_rank:
            low.append(("a1", d.decay_down.weight, d.decay_up.weight))
        if c.gate_rank:
            low.append(("g1", d.gate_down.weight, d.gate_up.weight))
        else:
            add("gate", d.gate_proj.weight)
        for n, down, _ in low:
            add(n, down)
        # the window's q | k | v and the delta rule's q | k | v are read as unpadded rows: only a block's start is aligned
        groups, at, self.at = [["wq", "wk", "wv"], ["q", "k", "v"]], 0, {}
        sizes = dict(zip(names, (w.shape[0] for w in ws)))
        for n in names:
            if not any(n in g[1:] for g in groups):
                at = up(at, 8)
            self.at[n] = at
            at += sizes[n]
        self.n_raw, self.act_cols = up(sum(w.shape[0] for w in raw), 128), up(at, 128)
        self.w_in = torch.cat((pad(torch.cat(raw, 0), self.n_raw, wp),
                               _stack_rows(ws, [self.at[n] for n in names], self.act_cols, wp)), 0)
        # second factors: [decay logits (fp32) | gate (bf16)] over [a1 | g1]
        self.low = None
        if low:
            k0 = self.at[low[0][0]]
            kc = up(self.at[low[-1][0]] + low[-1][1].shape[0] - k0, 8)
            assert k0 + kc <= self.act_cols
            nz = up(c.decays, 128) if c.decay_rank else 0
            ng = up(c.heads * c.vdim, 128) if c.gate_rank else 0
            w2 = torch.zeros(nz + ng, kc, dtype=ws[0].dtype, device=ws[0].device)
            for n, _, second in low:
                r0, k = (0 if n == "a1" else nz), self.at[n] - k0
                w2[r0:r0 + second.shape[0], k:k + second.shape[1]] = second.detach()
            self.low = types.SimpleNamespace(k0=k0, kc=kc, nz=nz, ng=ng, w=w2)
        self.taps, self.A_log, self.dt_bias = d.conv().detach().contiguous(), d.A_log.detach(), d.dt_bias.detach()
        self.o_norm, self.eps = d.o_norm.detach(), cfg.norm_eps
        self.o_cols = up(c.heads * c.vdim, 8)
        self.w_o = pad(d.o_proj.weight.detach(), wp, self.o_cols)
        self.norm1 = f32(layer.norm1.weight)
        self.moe = None
        if layer.mlp is not None:
            self._experts(layer.mlp, wp)
            self.norm2 = f32(layer.norm2.weight)

    def _experts(self, m, wp: int) -> None:
        c = m.cfg
        ff, W = up(c.ff, 64), m.w_down.shape[1]
        wd = up(W, 128)
        gu = torch.cat([_interleave(m.w_gate[e].detach(), m.w_up[e].detach(), ff, wp) for e in range(c.experts)], 0)
        dn = torch.zeros(c.experts, wd, ff, dtype=gu.dtype, device=gu.device)
        dn[:, :W, : c.ff] = m.w_down.detach()
        self.moe = types.SimpleNamespace(E=c.experts, top=c.top, ff=ff, wd=wd, up=gu, down=dn.view(c.experts * wd, ff),
                                         table=m.table.contiguous(), shared=None)
        if c.shared_ff:
            sf = up(c.shared_ff, 64)
            self.moe.shared = types.SimpleNamespace(
                ff=sf, up=_interleave(m.shared_gate.weight.detach(), m.shared_up.weight.detach(), sf, wp),
                down=pad(m.shared_down.weight.detach(), wp, sf))


class HybridStack:
    """Weights of the whole decoder, prepared once, and the launch sequence over them."""

    def __init__(self, model, device):
        cfg = model.config
        self.cfg, self.device = cfg, torch.device(device)
        self.width, self.wp = cfg.hidden_size, up(cfg.hidden_size, 8)
        self.layers = [_LayerWeights(l, cfg, i, self.wp) for i, l in enumerate(model.model.layers)]
        self.final_norm = model.model.norm.weight.detach().float().contiguous()
        table, head = model.model.embed_tokens.weight.detach(), model.lm_head.weight.detach()
        self.table, self.head = (w if self.wp == self.width else pad(w, w.shape[0], self.wp) for w in (table, head))
        self.vocab = cfg.vocab_size
        self.routed = [L for L in self.layers if L.moe is not None]
        self.side = torch.cuda.Stream(self.device) if self.device.type == "cuda" else None
        self.pass_rows = MAX_SORT_PAIRS // max([L.moe.top for L in self.routed], default=1)

    @staticmethod
    def caches(pool):
        """What :meth:`run` needs of a pool."""
        return pool

    # ------------------------------------------------------------------ buffers
    def buffers(self, T: int, max_keys: int) -> "types.SimpleNamespace":
        """Activation buffers for ``T`` rows; ``max_keys`` bounds a sequence's cache length (key splits)."""
        dev, cols = self.device, {}
        b = types.SimpleNamespace(T=T, max_keys=max_keys, cols=cols, ws={}, delta={})
        b.x = torch.zeros(T, self.wp, dtype=torch.float32, device=dev)
        b.h = torch.zeros(T, self.wp, dtype=torch.bfloat16, device=dev)
        # permutations of every routed layer: per pass [token of row | row of pair | group offsets]
        b.sort_off, at, passes = [], 0, (T + self.pass_rows - 1) // self.pass_rows
        rec = np.zeros(len(self.routed), dtype=_TABLE_LAYER)
        for j, L in enumerate(self.routed):
            rec[j] = (L.moe.table.data_ptr(), L.moe.top, L.moe.E, at, 0)
            b.sort_off.append(at)
            at += 2 * T * L.moe.top + passes * (L.moe.E + 1)
        if self.routed:
            b.sort_layers = torch.from_numpy(rec.view(np.uint8).reshape(-1).copy()).to(dev)
            b.sort = torch.empty(at, dtype=torch.int32, device=dev)

        def get(name, c, dtype=torch.bfloat16, rows=T, zero=False):
            key = (name, c, rows)
            if key not in cols:
                cols[key] = (torch.zeros if zero else torch.empty)(rows, c, dtype=dtype, device=dev)
            return cols[key]
        b.get = get
        return b

    def _delta_buf(self, st, L, hold: bool, kind: str = "rows", seqs: int = 0) -> dict:
        """Workspace of a delta layer: one for all layers of a shape, or one each when it has to outlive the forward."""
        c = L.dc
        key = L.index if hold else (kind, seqs, c.heads, c.kv_heads, c.dim, c.vdim, c.decays)
        if key not in st.delta:
            st.delta[key] = (X.delta_block_buffers(st.T, seqs, c, self.device) if kind == "blocks"
                             else X.delta_buffers(st.T, c, self.device))
        return st.delta[key]

    def _act(self, st, L, hold: bool) -> torch.Tensor:
        return st.get(f"act{L.index}" if hold else "act", L.act_cols)

    def _beside(self, fork: bool, side, main) -> int:
        """Launch ``side`` and ``main`` (functions of ``pdl for the first kernel``, returning launch counts), on two streams
        when ``fork``; everything launched later waits for both."""
        if not fork:
            return side(True) + main(True)
        cur = torch.cuda.current_stream()
        self.side.wait_stream(cur)
        with torch.cuda.stream(self.side):
            n = side(False)               # a plain dependency across streams
        n += main(True)
        cur.wait_stream(self.side)
        return n

    # ------------------------------------------------------------------ one forward
    def run(self, st, ids, pool, batch, xn, taps=None, tap_ids=None, pdl: bool = True) -> int:
        """Embed ``ids (T,)`` int32 and run every layer on ``st``; ``xn (T, wp)`` gets the final norm's output.  Returns
        the number of kernels launched."""
        lib, p, s = X.load(), X._p, X._stream
        T, n = st.T, 1
        X._check(lib.js_embed_f32(p(ids), p(self.table), self.vocab, self.table.stride(0), p(st.x), p(st.h), self.wp, T, self.width,
                                  int(pdl), s()), "js_embed_f32")
        if self.routed:
            X._check(lib.js_table_sort(p(st.sort_layers), len(self.routed), p(ids), T, self.pass_rows, self.vocab,
                                       max(L.moe.top for L in self.routed), max(L.moe.E for L in self.routed), p(st.sort), int(pdl), s()),
                     "js_table_sort")
            n += 1
        last = len(self.layers) - 1
        tap_ids = list(tap_ids) if taps is not None else []
        for i, L in enumerate(self.layers):
            tap = None
            if i in tap_ids and i != last:
                j = tap_ids.index(i)
                tap = taps[:, j * self.width:(j + 1) * self.width]
            n += self._layer(st, L, pool, batch, xn if i == last else None, tap, pdl)
        for j, t in enumerate(tap_ids):
            if t == last:
                taps[:, j * self.width:(j + 1) * self.width].copy_(xn[:, : self.width])
            elif tap_ids.index(t) != j:
                k = tap_ids.index(t)
                taps[:, j * self.width:(j + 1) * self.width].copy_(taps[:, k * self.width:(k + 1) * self.width])
        return n

    def _resid(self, st, w, eps, out, tap, pdl, ya=None, bias=None, wa=None, yb=None, wb=None, ys=None, inv=None, k=0, sh=None,
               t0: int = 0, rows=None) -> None:
        """The residual step on rows ``[t0, t0 + rows)``; ``out`` is the final norm's output where it is due."""
        p = X._p
        rows = st.T if rows is None else rows
        at = lambda t: X._vp(t.data_ptr() + t0 * t.stride(0) * t.element_size()) if t is not None else X._vp(0)
        ld = lambda t: t.stride(0) if t is not None else 0
        h = out if out is not None else st.h
        assert h.stride(0) == st.x.stride(0)
        X._check(X.load().js_resid_norm(
            at(ya), ld(ya), p(bias), p(wa), at(yb), ld(yb), p(wb), p(ys), ld(ys), p(inv), k, at(sh), ld(sh), p(w),
            p(self.final_norm if out is not None else None), X.ctypes.c_float(eps), at(st.x), at(h), self.wp, at(tap), ld(tap), rows,
            self.width, int(pdl), X._stream()), "js_resid_norm")

    def _layer(self, st, L, pool, batch, out, tap, pdl) -> int:
        c, hold = L.dc, batch.mask is not None
        raw, act = st.get("raw", L.n_raw, torch.float32), self._act(st, L, hold)
        X.gemm_inproj(st.h, L.w_in, raw, L.n_raw, act, False, pdl=pdl, act=X.ACT_NONE)
        n = 1
        b, z = raw[:, : c.heads], raw[:, c.heads:]
        if L.low is not None:
            z = st.get("z", L.low.nz, torch.float32) if L.low.nz else z
            gate = st.get("gate", L.low.ng) if L.low.ng else None
            X.gemm_inproj(act[:, L.low.k0:L.low.k0 + L.low.kc], L.low.w, z if L.low.nz else None, L.low.nz, gate, False, pdl=pdl,
                          act=X.ACT_NONE)
            n += 1
        if not c.gate_rank:
            gate = act[:, L.at["gate"]:]
        yl, yr = st.get("yl", self.wp), st.get("yr", self.wp)
        pre = act[:, L.at["q"]:L.at["q"] + c.channels]
        fork = L.parallel and self._forks(st)
        window = lambda first: self._window(st, L, pool, batch, act, yl, pdl, pdl and first) if L.parallel else 0
        n += self._beside(fork, window, lambda first: self._delta(st, L, pool, batch, pre, z, b, gate, yr, hold, pdl))
        mlp = L.moe is not None
        end = dict(out=None if mlp else out, tap=None if mlp else tap)
        if L.parallel:
            self._resid(st, L.norm1, L.eps, ya=yl, bias=L.win.o_bias, wa=L.left_norm, yb=yr, wb=L.right_norm, pdl=pdl and not fork, **end)
        else:
            self._resid(st, L.norm1, L.eps, ya=yr, pdl=pdl, **end)
        n += 1
        if mlp:
            n += self._experts(st, L, out, tap, pdl)
        return n

    def _forks(self, st) -> bool:
        return st.T >= FORK_MIN_TOKENS or torch.cuda.is_current_stream_capturing()

    def _window(self, st, L, pool, batch, act, y, pdl, first_pdl) -> int:
        o, n = L.win.run(st, pool.layer(L.index), batch, act[:, L.at["wq"]:], None, None, pdl, first_pdl)
        X.gemm(o, L.win.w_o, out=y, pdl=pdl)
        return n + 1

    def _delta(self, st, L, pool, batch, pre, z, b, gate, y, hold, pdl) -> int:
        c = L.dc
        state, conv = pool.states.layer(L.index)
        o = st.get("do", L.o_cols, zero=L.o_cols != c.heads * c.vdim)
        gate = gate[:, : c.heads * c.vdim]
        seqs = (batch.state_rows, batch.cu_q, batch.past)
        if hold:
            buf = self._delta_buf(st, L, True)
            X.delta_prep(buf, c, pre, z, b, L.taps, L.A_log, L.dt_bias, conv, *seqs, batch.mask, pdl=pdl)
            X.delta_seq(buf, c, state, conv, pre, *seqs, batch.mask, pdl=pdl)
            X.gated_head_norm(buf["o"], L.o_norm, gate, c.gate, L.eps, out=o, pdl=pdl)
            n = 3
        else:
            n = X.delta_forward(c, pre, z, b, L.taps, L.A_log, L.dt_bias, state, conv, *seqs, gate, L.o_norm, c.gate, L.eps, o,
                                batch.max_rows, buffers=lambda kind: self._delta_buf(st, L, False, kind, batch.state_rows.numel()), pdl=pdl)
        X.gemm(o, L.w_o, out=y, pdl=pdl)
        return n + 1

    def _experts(self, st, L, out, tap, pdl) -> int:
        m, T = L.moe, st.T
        fork = m.shared is not None and self._forks(st)
        a, sh = (st.get("sa", m.shared.ff), st.get("sh", self.wp)) if m.shared is not None else (None, None)
        pending = []

        def shared(first):
            if m.shared is None:
                return 0
            X.gemm(st.h, m.shared.up, out=a, epi=X.EPI_SWIGLU, pdl=pdl and first)
            X.gemm(a, m.shared.down, out=sh, pdl=pdl)
            return 2

        def routed(first):
            at = st.sort_off[self.routed.index(L)]
            for t0 in range(0, T, self.pass_rows):
                rows = min(self.pass_rows, T - t0)
                P = rows * m.top
                tok, inv, off = st.sort[at:at + P], st.sort[at + P:at + 2 * P], st.sort[at + 2 * P:at + 2 * P + m.E + 1]
                at += 2 * P + m.E + 1
                g = lambda name, c: st.get(f"{name}{t0}", c, rows=P)
                xs, hs, ys = g("xs", self.wp), g("hs", m.ff), g("ys", m.wd)
                X.gather_rows(st.h, tok, xs, pdl=pdl)
                cover = min(rows, ((4 * P // m.E + 128 + 127) // 128) * 128)
                X.gemm_grouped(xs, m.up, hs, P, 2 * m.ff, m.E, off, cover, X.EPI_SWIGLU)
                X.gemm_grouped(hs, m.down, ys, P, m.wd, m.E, off, cover, X.EPI_STORE)
                pending.append((ys, inv, t0, rows))
            return 3 * len(pending)

        n = self._beside(fork, shared, routed)
        pdl = pdl and not fork
        for ys, inv, t0, rows in pending:          # h is rewritten here, so every pass has read it first
            self._resid(st, L.norm2, L.eps, out, tap, pdl, ys=ys, inv=inv, k=m.top, sh=sh, t0=t0, rows=rows)
            n += 1
        return n

    # ------------------------------------------------------------------ token trees
    def commit(self, st, pool, state_rows, cu_q, past, path, path_len, pdl: bool = True) -> int:
        """Advance one sequence's states along the rows ``path[:path_len]`` (device) of the tree forward run on ``st``;
        ``past`` is the committed length behind the path."""
        for L in self.layers:
            state, conv = pool.states.layer(L.index)
            pre = self._act(st, L, True)[:, L.at["q"]:L.at["q"] + L.dc.channels]
            X.delta_seq(self._delta_buf(st, L, True), L.dc, state, conv, pre, state_rows, cu_q, past, path=path, path_len=path_len, pdl=pdl)
        return len(self.layers)

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
                                     mask=None if causal or max_q == 1 else mask, positions=positions, max_keys=max_keys,
                                     max_rows=max_q, state_rows=seq_rows if state_rows is None else state_rows)

    def ragged_batch(self, slot_map, meta, counts, past_lens):
        """Portions of prompts beside decoded tokens, or token trees."""
        return types.SimpleNamespace(slot_map=slot_map, seq_rows=meta.seq_rows, cu_q=meta.cu_q, past=meta.past_lens, slots=meta.slots,
                                     mask=None if meta.causal else meta.mask_bits, positions=meta.positions,
                                     max_keys=max(a + b for a, b in zip(counts, past_lens)), max_rows=max(counts),
                                     state_rows=meta.seq_rows)
