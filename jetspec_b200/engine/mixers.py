"""Fused kernel forms of single mixers for the engine's launch sequences: kernel-ready weights, and everything between a layer's
input GEMM and its output GEMM.  :mod:`~jetspec_b200.engine.latent_stack`, :mod:`~jetspec_b200.engine.hybrid_stack` and
:mod:`~jetspec_b200.engine.prenorm_stack` put them together.

Every size is padded to what the kernels want when the weights are prepared; padding is zero and stays zero.
"""
from __future__ import annotations

import torch

from ..ops import cuda_ext as X
from ..runtime.kv_pool import latent_row_width, window_row_width

EXPAND_MIN_TOKENS = 128       # a portion of at least this many tokens may take the expanded form of latent attention


def up(n: int, m: int) -> int:
    return (int(n) + m - 1) // m * m


def pad(w: torch.Tensor, rows: int, cols: int) -> torch.Tensor:
    if w.shape == (rows, cols):
        return w.contiguous()
    out = torch.zeros(rows, cols, dtype=w.dtype, device=w.device)
    out[: w.shape[0], : w.shape[1]] = w
    return out


def pad_heads(w: torch.Tensor, heads: int, rows: int, cols: int) -> torch.Tensor:
    """``(heads * r, c)`` -> ``(heads * rows, cols)``, every head padded on its own."""
    r = w.shape[0] // heads
    out = torch.zeros(heads, rows, cols, dtype=w.dtype, device=w.device)
    out[:, :r, : w.shape[1]] = w.view(heads, r, w.shape[1])
    return out.view(heads * rows, cols)


def split_ws(st, splits: int, rows: int, cols: int):
    """Partial outputs and (maximum, sum) pairs of an attention launch with several key splits."""
    if splits == 1:
        return None
    key = (splits, rows, cols)
    if key not in st.ws:
        dev = st.x.device
        st.ws[key] = {"o": torch.zeros(splits, rows, cols, dtype=torch.float32, device=dev),
                      "ml": torch.zeros(splits, rows, 2, dtype=torch.float32, device=dev)}
    return st.ws[key]


class WindowMixer:
    """Attention over K/V pools, in a window or over the whole past: one kernel behind the input projections (biases, norms,
    rotation, temperature, cache scatter), the means of blocks that are whole by then where the layer pools blocks, then the
    tcgen05 attention (heads up to 128, groups of up to 16) or the plain-core one; sinks, gates, capped scores, pooled blocks and
    the difference of two maps ride in its softmax and epilogue.  ``proj`` are the unpadded q | k | v columns (q | k where the
    values are the keys, q alone over another layer's), ``gate`` one fp32 logit per (padded) head."""

    def __init__(self, m, eps: float, wp: int):
        c = self.cfg = m.cfg
        f32 = lambda p: p.detach().float().contiguous()
        g = c.heads // c.kv_heads
        self.eps = eps
        self.Dp, self.Vp = window_row_width(c.dim, c.vdim, torch.bfloat16, c.maps)
        gp = 1 << (g - 1).bit_length()
        # what the tensor-core kernel takes
        self.tc = self.Dp == 128 and self.Vp == 128 and gp <= 16 and X.window_tc_ok(c.maps, c.pool, c.softcap)
        self.gp, self.Dq, self.vq = (gp, 128 // c.maps, 128) if self.tc else (g, c.dim, c.vdim)
        self.heads = c.kv_heads * self.gp
        self.q_cols, self.o_cols = self.heads * c.maps * self.Dq, up(self.heads * self.vq, 8)
        w = m.o_proj.weight.detach()
        o = torch.zeros(wp, c.kv_heads, self.gp, self.vq, dtype=w.dtype, device=w.device)
        o[: w.shape[0], :, :g, : c.vdim] = w.view(-1, c.kv_heads, g, c.vdim)
        self.w_o = pad(o.view(wp, -1), wp, self.o_cols)
        projs = [p for p in (m.q_proj, m.k_proj, m.v_proj) if p is not None]
        self.qkv_bias = torch.cat([f32(p.bias) for p in projs]) if c.bias else None
        self.o_bias = f32(m.o_proj.bias) if m.o_proj.bias is not None else None
        self.qkv = [p.weight.detach() for p in projs]
        self.v_col = (c.heads + (0 if c.tie_values else c.kv_heads)) * c.maps * c.dim
        self.q_norm, self.k_norm = (f32(m.q_norm), f32(m.k_norm)) if c.proj_norm else (None, None)
        self.freq = X.pair_freq(c.rot_dims, c.rot_base, w.device) if c.rot is None else None
        self.sink, self.gate = c.sink, None
        if c.sink_logits:
            self.sink = pad_heads(f32(m.sink_logits).view(-1, 1), c.kv_heads, self.gp, 1).view(-1).contiguous()
        if c.gate:
            self.gate = pad_heads(m.gate_proj.weight.detach(), c.kv_heads, self.gp, m.gate_proj.weight.shape[1])
        self.diff = m.differential()
        if self.diff is not None:
            self.diff = (self.diff[0].detach().reshape(1).contiguous(), *self.diff[1:])

    def run(self, st, pool, batch, proj, gate, rot, pdl: bool, first_pdl: bool, blocks=None):
        """Returns the attention output ``(T, o_cols)`` and the number of kernels launched."""
        c, T = self.cfg, st.T
        lib, p = X.load(), X._p
        kp, vp = pool
        q = st.get("wq", self.q_cols, zero=self.heads != c.heads)
        status = p(X.status_word(kp.device))
        if c.rot is None:
            X._check(lib.js_window_post(
                p(proj), proj.stride(0), p(self.qkv_bias), c.heads, c.kv_heads, self.gp, c.maps, c.dim, c.vdim, self.Dq, self.Dp, self.Vp,
                c.rot_dims, p(self.freq), int(c.qk_norm), X.ctypes.c_float(self.eps), c.temp_every, X.ctypes.c_float(c.temp_coef), self.v_col,
                int(c.kv_from is None), p(batch.positions), p(batch.slots), kp.shape[1], T, p(q), p(kp), p(vp), status, int(first_pdl),
                X._stream()), "js_window_post")
        else:
            X._check(lib.js_attn_post(
                p(proj), proj.stride(0), p(self.qkv_bias), p(self.q_norm), p(self.k_norm), c.heads, c.kv_heads, self.gp, c.dim, c.vdim, self.Dq,
                self.Dp, self.Vp, c.rot.dims, int(c.rot.pairing == "next"), p(rot), rot.stride(0) // 2, X.ctypes.c_float(self.eps),
                p(batch.slots), kp.shape[1], T, p(q), p(kp), p(vp), status, int(first_pdl), X._stream()), "js_attn_post")
        o = st.get("wo", self.o_cols, zero=True)
        Hq, n = self.heads, 2
        if blocks is not None and batch.mask is None:        # rows of a token tree are not committed yet
            X.pool_blocks(kp, vp, *blocks, batch.slot_map, batch.seq_rows, batch.cu_q, batch.past, rows=T, pdl=pdl)
            n += 1
        args = (batch.slot_map, batch.seq_rows, batch.cu_q, batch.past, batch.mask)
        more = dict(keep_first=c.keep_first, gate=gate)
        if c.softcap or blocks is not None or self.diff is not None:
            more.update(softcap=c.softcap, blocks=blocks, diff=self.diff)
        # a token tree deeper than the window would see blocks of its own nodes, which only the plain-core kernel makes
        shallow = batch.mask is None or (batch.mask.shape[1] <= 8 and (blocks is None or c.window >= batch.max_rows))
        if self.tc and shallow:
            if self.diff is not None:
                more.update(vdim=c.vdim)
            splits = X.window_attn_splits(T, Hq, c.kv_heads, batch.max_keys, c.window, c.keep_first, c.pool, batch.seq_rows.numel())
            X.window_attention_tc(q.view(T, Hq, 128), kp, vp, *args, c.scale, c.window, self.sink, batch.mask is None, o, splits=splits,
                                  ws=split_ws(st, splits, T * Hq * c.maps, 128), pdl=pdl, **more)
            n += int(splits > 1 and (self.diff is not None or not X.attn_merges_in_cluster(T, Hq, c.kv_heads, splits)))
        else:
            X.window_attention(q.view(T, Hq * c.maps, self.Dq), kp, vp, self.vq, *args, c.scale, c.window, self.sink, batch.mask is None, out=o,
                               pdl=pdl, norm_dim=c.vdim, **more)
        return o, n


class LatentMixer:
    """Latent attention over paged latent rows, in one of two forms:

    *absorbed* (decode, trees, short portions): ``W_uk`` is applied to the query and ``W_uv`` behind the attention, both as batched
    GEMMs over heads, and the tcgen05 latent kernel attends over the cached rows themselves;
    *expanded* (long prompt portions): keys and values are expanded from the gathered rows once and the tcgen05 K/V kernel
    attends over them, which costs (dim + vdim) instead of 2 kv_rank per score.

    A rotated key part simply lengthens the heads and the cached row: the products that map queries and rows carry an
    identity block for it, and only the latent's own columns are values."""

    def __init__(self, mix):
        m = self.cfg = mix.cfg
        H, dim = m.heads, m.dim + m.rot_dim
        self.rp, self.vk = latent_row_width(m.row), latent_row_width(m.kv_rank)
        # the K/V kernel has 128-wide heads; padding narrower ones up to it pays from 64 on
        self.expand = 64 <= dim <= 128 and 64 <= m.vdim <= 128
        self.dp, self.vp = (128, 128) if self.expand else (up(dim, 8), up(m.vdim, 8))
        self.out_cols = H * self.vp
        uk, uv = mix.k_up.weight.detach(), mix.v_up.weight.detach()
        full = torch.zeros(H, dim, m.row, dtype=uk.dtype, device=uk.device)       # a cached row to every head's key
        full[:, : m.dim, : m.kv_rank] = uk.view(H, m.dim, m.kv_rank)
        full[:, m.dim:, m.kv_rank:] = torch.eye(m.rot_dim, dtype=uk.dtype, device=uk.device)
        self.uk_t = pad_heads(full.transpose(1, 2).reshape(H * m.row, dim), H, self.rp, self.dp)
        self.uv = pad_heads(uv, H, self.vp, self.vk)
        # keys and values of every head from a cached row, one product: [heads * 128 keys | heads * 128 values]
        self.ukv = None
        if self.expand:
            self.ukv = torch.cat((pad_heads(full.view(H * dim, m.row), H, self.dp, self.rp), pad_heads(uv, H, self.vp, self.rp)), 0)
        self.sinks = mix.sink.detach().float().contiguous() if mix.sink is not None else None
        o = mix.o_proj.weight.detach()
        self.w_o = torch.zeros(o.shape[0], H, self.vp, dtype=o.dtype, device=o.device)
        self.w_o[:, :, : m.vdim] = o.view(-1, H, m.vdim)
        self.w_o = self.w_o.view(-1, self.out_cols)

    def attend(self, st, pool, batch, q, out, gate, pdl: bool) -> int:
        """Attention of ``q (T, heads * dp)`` for every part of the batch, to the first ``out_cols`` columns of ``out``."""
        n = 0
        for part in batch.parts:
            n += (self._expanded if part.expand and self.expand else self._absorbed)(st, pool, batch, part, q, out, gate, pdl)
        return n

    def _absorbed(self, st, pool, batch, part, q, out, gate, pdl) -> int:
        r0, r1, H, m = part.r0, part.r1, self.cfg.heads, self.cfg
        T = r1 - r0
        qa, ol = st.get("qa", H * self.rp)[r0:r1], st.get("ol", H * self.rp)[r0:r1]
        X.gemm_batched(q[r0:r1], self.uk_t, qa, H, self.rp, self.dp, self.dp, self.rp, H * self.rp, pdl=pdl)
        rows = T * H
        tc = X.latent_tc_ok(self.rp, self.vk) and (batch.mask is None or batch.mask.shape[1] <= 8)
        splits = X.latent_attn_splits(T, H, part.seqs, part.max_q, self.rp, part.max_keys, self.vk) if tc else 1
        X.latent_attention_rows(qa.view(rows, self.rp), pool, H, batch.slot_map, part.seq_rows, part.cu_q, part.past,
                                None if batch.mask is None else batch.mask[r0:r1], m.scale, batch.mask is None, part.max_q,
                                out=ol.view(rows, self.rp), splits=splits, ws=split_ws(st, splits, rows, self.rp), pdl=pdl,
                                impl="tc" if tc else "simt", out_cols=self.vk, sinks=self.sinks, gate=None if gate is None else gate[r0:r1])
        X.gemm_batched(ol, self.uv, out[r0:r1], H, self.vp, self.vk, self.rp, self.vp, out.stride(0), pdl=pdl)
        return 4 if splits > 1 else 3

    def _expanded(self, st, pool, batch, part, q, out, gate, pdl) -> int:
        r0, r1, H, keys = part.r0, part.r1, self.cfg.heads, part.keys
        c, kv = st.get("c", self.rp, rows=keys), st.get("kv", H * 256, rows=keys)
        X.gather_rows(pool, part.key_slots, c, pdl=pdl)
        X.gemm(c, self.ukv, out=kv, pdl=pdl)
        X.paged_attention_rows(q[r0:r1].view(r1 - r0, H, 128), kv[:, : H * 128], kv[:, H * 128:], part.key_map, part.key_base, part.cu_q,
                               part.past, self.cfg.scale, part.max_q, out[r0:r1], part.max_keys, pdl=pdl, sinks=self.sinks,
                               gate=None if gate is None else gate[r0:r1])
        return 3


class RetentionMixer:
    """Retention: rotation to gated norm in one kernel (decode steps, token trees) or three (portions); ``act`` are the q | k | v |
    gate columns, each block aligned to 8."""

    def __init__(self, m, eps: float, wp: int):
        c = self.cfg = m.cfg
        self.eps = eps
        self.weights = [p.weight.detach() for p in (m.q_proj, m.k_proj, m.v_proj, m.gate_proj)]
        at, self.offs = 0, []
        for w in self.weights:
            self.offs.append(at)
            at = up(at + w.shape[0], 8)
        self.act_cols, self.cols = at, tuple(self.offs[1:])
        if self.cols[0] != up(c.heads * c.dim, 8):
            raise AssertionError("q starts the block")
        self.o_cols = up(c.heads * c.vdim, 8)
        self.w_o = pad(m.o_proj.weight.detach(), wp, self.o_cols)
        X.retention_powers(c, m.o_proj.weight.device)          # made here: a captured launch must not copy from the host

    def run(self, st, state, batch, act, rot, pdl: bool):
        """Returns the output ``(T, o_cols)`` and the number of kernels launched."""
        c, dev = self.cfg, act.device
        o = st.get("ro", self.o_cols, zero=self.o_cols != c.heads * c.vdim)

        def buffers(kind):
            seqs = batch.state_rows.numel()
            key = ("retention", kind, seqs, c.heads, c.dim, c.vdim)
            if key not in st.ws:
                st.ws[key] = (X.retention_chunk_buffer(st.T, seqs, c, dev) if kind == "chunks" else X.retention_rows_buffers(st.T, c, dev))
            return st.ws[key]
        n = X.retention_forward(c, act, self.cols, rot, state, batch.state_rows, batch.cu_q, batch.past, batch.mask, self.eps, o, batch.max_rows,
                                buffers=buffers, pdl=pdl)
        return o, n

    def advance(self, act, rot, state, state_rows, cu_q, past, path, path_len, pdl: bool) -> None:
        X.retention_path(self.cfg, act, self.cols, rot, state, state_rows, cu_q, past, path, path_len, pdl=pdl)
