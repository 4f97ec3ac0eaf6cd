"""Fused kernel form of a decoder of parallel latent-attention blocks (Karuzen) for the engine's kernel path.

Per layer run, with everything between the GEMMs folded into them or into one small kernel:

1. ONE input GEMM on the normalised stream ``h``: the two latents' down-projections, the router and the shared expert's
   gate leave as fp32; gate/up (or the shared expert's up) leave as activated bf16, next to where the attention output
   will be (``cat``);
2. latent RMS norms, the new row goes straight to its pool slot; sigmoid routing scales the shared activations;
3. query up-projection, then one of the two attention forms of :class:`~jetspec_b200.engine.mixers.LatentMixer`;
4. ONE output GEMM over ``cat``: attention output and feed-forward are both added to the fp32 residual stream, and the
   NEXT run's Dynamic Tanh is applied in the epilogue (with the embedding added first where a loop pass begins).
   Routed layers apply it in the experts' combine kernel instead.

Every size is padded to what the kernels want when the weights are prepared; padding is zero and stays zero.
"""
from __future__ import annotations

import types

import torch

from ..ops import cuda_ext as X
from .mixers import EXPAND_MIN_TOKENS, LatentMixer, pad, pad_heads, up

MAX_SORT_PAIRS = 16384        # (token, expert) pairs one launch of the permutation kernel takes


class _LayerWeights:
    """Kernel-ready weights of one layer (shared by its runs)."""

    def __init__(self, layer, width: int, wp: int):
        m, mix, mlp = layer.mixer.cfg, layer.mixer, layer.mlp
        self.q_rank, self.kv_rank, self.eps = m.q_rank, m.kv_rank, mix.eps
        self.mix = LatentMixer(mix)
        self.qp = up(m.q_rank, 8)
        self.norm = (layer.norm.weight.float(), layer.norm.bias.float(), layer.norm.alpha.item())
        self.q_norm, self.kv_norm = mix.q_norm, mix.kv_norm
        raw = [mix.q_down.weight, mix.kv_down.weight]
        self.moe = None
        act_w = None
        self.act_cols = 0
        self.gelu = True
        if mlp is not None and hasattr(mlp, "gate_proj"):
            ff = up(mlp.gate_proj.weight.shape[0], 64)
            g, u = (pad(w, ff, width).view(ff // 64, 64, width) for w in (mlp.gate_proj.weight, mlp.up_proj.weight))
            act_w, self.act_cols, down = torch.cat((g, u), 1).reshape(2 * ff, width), ff, mlp.down_proj.weight
        elif mlp is not None:
            c = mlp.cfg
            raw.append(mlp.router.weight)
            ffp, wd = up(c.ff, 128), up(width, 128)
            self.moe = types.SimpleNamespace(
                E=c.experts, top=c.top, scale=c.scale, ffp=ffp, wd=wd, corr=mlp.correction.float().contiguous(),
                up=torch.zeros(c.experts * ffp, wp, dtype=mlp.w_up.dtype, device=mlp.w_up.device),
                down=torch.zeros(c.experts * wd, ffp, dtype=mlp.w_up.dtype, device=mlp.w_up.device),
                z_col=m.q_rank + m.kv_rank, gate_col=-1)
            self.moe.up.view(c.experts, ffp, wp)[:, : c.ff, :width] = mlp.w_up
            self.moe.down.view(c.experts, wd, ffp)[:, :width, : c.ff] = mlp.w_down
            if c.shared_ff:
                raw.append(mlp.shared_gate.weight)
                self.moe.gate_col = c.experts
                self.gelu, self.act_cols = False, up(c.shared_ff, 128)
                act_w, down = pad(mlp.shared_up.weight, self.act_cols, width), mlp.shared_down.weight
        raw_w = torch.cat(raw, 0)
        self.n_raw = up(raw_w.shape[0], 128)
        raw_w = pad(raw_w, self.n_raw, width)
        self.w_in = pad(raw_w if act_w is None else torch.cat((raw_w, act_w), 0), self.n_raw + (0 if act_w is None else act_w.shape[0]), wp)
        self.uq = pad(pad_heads(mix.q_up.weight, m.heads, self.mix.dp, m.q_rank), m.heads * self.mix.dp, self.qp)
        attn_cols = self.mix.out_cols
        self.cat_cols = attn_cols + self.act_cols
        self.w_out = torch.zeros(wp, self.cat_cols, dtype=mix.o_proj.weight.dtype, device=mix.o_proj.weight.device)
        self.w_out[:width, :attn_cols] = self.mix.w_o
        self.mix.w_o = None
        if self.act_cols:
            self.w_out[:width, attn_cols:attn_cols + down.shape[1]] = down


class LatentStack:
    """Weights of the whole decoder, prepared once, and the launch sequence over them."""

    def __init__(self, model, device):
        cfg = model.config
        self.cfg, self.device = cfg, torch.device(device)
        self.width, self.wp = cfg.hidden_size, up(cfg.hidden_size, 8)
        self.layers = [_LayerWeights(l, self.width, self.wp) for l in model.model.layers]
        for L in self.layers:
            L.norm = self._pad_norm(*L.norm)
        fn = model.model.norm
        self.final_norm = self._pad_norm(fn.weight.float(), fn.bias.float(), fn.alpha.item())
        self.runs = cfg.layer_runs()
        table = model.model.embed_tokens.weight
        self.table = table if self.wp == self.width else pad(table, table.shape[0], self.wp)
        self.head = self.table
        self.vocab = cfg.vocab_size
        self.loops = any(again for _, again in self.runs)

    def _pad_norm(self, w, b, alpha):
        p = lambda v: pad(v.view(1, -1), 1, self.wp).view(-1)
        return p(w), p(b), alpha

    @staticmethod
    def caches(pool):
        """What :meth:`run` needs of a pool."""
        return pool.latent_pools

    # ------------------------------------------------------------------ buffers
    def buffers(self, T: int, max_keys: int) -> "types.SimpleNamespace":
        """Activation buffers for ``T`` rows; ``max_keys`` bounds a sequence's cache length (key splits)."""
        dev, cols = self.device, {}
        b = types.SimpleNamespace(T=T, max_keys=max_keys, cols=cols)
        bf = lambda n, c: torch.zeros(n, c, dtype=torch.bfloat16, device=dev)
        b.x = torch.zeros(T, self.wp, dtype=torch.float32, device=dev)
        b.emb = bf(T, self.wp) if self.loops else None
        b.h = bf(T, self.wp)
        b.ws = {}

        def get(name, c, dtype=torch.bfloat16, rows=T):
            key = (name, c, rows)
            if key not in cols:
                cols[key] = torch.empty(rows, c, dtype=dtype, device=dev)
            return cols[key]
        b.get = get
        return b

    # ------------------------------------------------------------------ one forward
    def run(self, st, ids, pools, batch, xn, taps=None, tap_ids=None, pdl: bool = True) -> int:
        """Embed ``ids (T,)`` int32 and run every layer on ``st``; ``xn (T, wp)`` gets the final norm's output.

        ``batch``: ``slot_map, slots, mask, causal`` of the ragged batch and ``parts``, its sequence groups in row
        order (see :meth:`part`).  Returns the number of kernels launched."""
        T, n = st.T, 1
        tap_ids = list(tap_ids) if taps is not None else []
        nw, nb, alpha = self.layers[self.runs[0][0]].norm
        lib, p, s = X.load(), X._p, X._stream
        X._check(lib.js_embed_dyt(p(ids), p(self.table), self.vocab, self.table.stride(0), p(st.x), p(st.emb), p(st.h), self.wp,
                                  p(nw), p(nb), X.ctypes.c_float(alpha), T, self.width, int(pdl), s()), "js_embed_dyt")
        last = len(self.runs) - 1
        for r, (i, _) in enumerate(self.runs):
            L = self.layers[i]
            again = r < last and self.runs[r + 1][1]
            norm, h = (self.final_norm, xn) if r == last else (self.layers[self.runs[r + 1][0]].norm, st.h)
            tapped = r in tap_ids and r != last
            n += self._layer(st, L, pools[r], batch, norm, h, st.emb if again else None, tapped, pdl)
            if tapped:
                for j, t in enumerate(tap_ids):
                    if t == r:
                        X._check(lib.js_tap_rows(p(st.x), self.wp, X._vp(taps.data_ptr() + 2 * j * self.width), taps.stride(0), T,
                                                 self.width, int(pdl), s()), "js_tap_rows")
                        n += 1
                self._combine(st, None, st.emb if again else None, norm, h, pdl)
                n += 1
        if last in tap_ids:
            for j, t in enumerate(tap_ids):
                if t == last:
                    taps[:, j * self.width:(j + 1) * self.width].copy_(xn[:, : self.width])
        return n

    def _combine(self, st, moe, emb, norm, h, pdl):
        """Residual tail: routed experts' weighted rows, the embedding of a loop pass, the next norm."""
        lib, p = X.load(), X._p
        nw, nb, alpha = norm if norm is not None else (None, None, 0.0)
        ys, inv, row_w, k, t0, rows = moe if moe is not None else (None, None, None, 0, 0, st.T)
        off = lambda t: X._vp(t.data_ptr() + t0 * t.stride(0) * t.element_size()) if t is not None else X._vp(0)
        X._check(lib.js_combine_dyt(p(ys), ys.stride(0) if ys is not None else 0, p(inv), p(row_w), k, off(emb), off(st.x),
                                    off(h) if norm is not None else X._vp(0), self.wp, p(nw), p(nb), X.ctypes.c_float(alpha), rows,
                                    self.wp, int(pdl), X._stream()), "js_combine_dyt")

    def _layer(self, st, L, pool, batch, norm, h, emb, tapped, pdl) -> int:
        lib, p, s = X.load(), X._p, X._stream
        T, mix = st.T, L.mix
        raw, cat = st.get("raw", L.n_raw, torch.float32), st.get("cat", L.cat_cols)
        act = cat[:, mix.out_cols:] if L.act_cols else None
        X.gemm_inproj(st.h, L.w_in, raw, L.n_raw, act, L.gelu, pdl=pdl)
        n = 1
        pending = []
        if L.moe is not None:
            pending, launched = self._experts(st, L, raw, act, pdl)
            n += launched
        cq, q = st.get("cq", L.qp), st.get("q", mix.cfg.heads * mix.dp)
        X._check(lib.js_latent_post(p(raw), L.n_raw, L.q_rank, L.kv_rank, p(L.q_norm), p(L.kv_norm), X.ctypes.c_float(L.eps), p(cq),
                                    L.qp, p(pool), mix.rp, pool.shape[0], p(batch.slots), T, p(X.status_word(self.device)),
                                    int(pdl), s()), "js_latent_post")
        X.gemm(cq, L.uq, out=q, pdl=pdl)
        n += 2 + mix.attend(st, pool, batch, q, cat, None, pdl)
        # the norm rides on the output GEMM unless a kernel still has to add to the stream (experts) or read it (taps)
        fused = not pending and not tapped
        X.gemm_resid32(cat, L.w_out, st.x, norm=norm if fused else None, h=h if fused else None, emb=emb if fused else None, pdl=pdl)
        n += 1
        for moe in pending:
            self._combine(st, moe, None if tapped else emb, None if tapped else norm, h, pdl)
            n += 1
        return n

    def _experts(self, st, L, raw, act, pdl):
        """Route, sort by expert, run the two grouped GEMMs; the weighted rows stay behind for :meth:`_combine`."""
        m, T = L.moe, st.T
        wts, idx = st.get("wts", m.top, torch.float32), st.get("idx", m.top, torch.int32)
        X.sigmoid_route(raw[:, m.z_col:], m.corr, m.top, m.scale, m.gate_col, act, wts=wts, idx=idx, pdl=pdl)
        lib, p, s = X.load(), X._p, X._stream
        step = max(1, MAX_SORT_PAIRS // m.top)
        pending, n = [], 1
        for t0 in range(0, T, step):
            rows = min(step, T - t0)
            P = rows * m.top
            g = lambda name, c, dt=torch.bfloat16: st.get(f"{name}{t0}", c, dt, rows=P)
            order, tok, inv = (st.get(f"{k}{t0}", P, torch.int32, rows=1) for k in ("order", "tok", "inv"))
            row_w, off = st.get(f"row_w{t0}", P, torch.float32, rows=1), st.get(f"off{t0}", m.E + 1, torch.int32, rows=1)
            cnt = st.get(f"cnt{t0}", m.E, torch.int32, rows=1)
            X._check(lib.js_moe_sort_inv(p(idx[t0:]), p(wts[t0:]), P, m.E, 0, m.E, p(order), p(row_w), p(off), p(cnt), m.top, p(tok),
                                         p(inv), int(pdl), s()), "js_moe_sort_inv")
            xs, hs, ys = g("xs", self.wp), g("hs", m.ffp), g("ys", m.wd)
            X.gather_rows(st.h[t0:t0 + rows], tok.view(-1), xs, pdl=pdl)
            cover = min(rows, ((4 * P // m.E + 128 + 127) // 128) * 128)
            X.gemm_grouped(xs, m.up, hs, P, m.ffp, m.E, off, cover, X.EPI_RELU2)
            X.gemm_grouped(hs, m.down, ys, P, m.wd, m.E, off, cover, X.EPI_STORE)
            pending.append((ys, inv, row_w, m.top, t0, rows))
            n += 4
        return pending, n

    # ------------------------------------------------------------------ batches
    def uniform_batch(self, slot_map, seq_rows, cu_q, past, slots, mask, causal, rows, max_q, max_keys, positions=None,
                      state_rows=None):
        """A batch whose sequences all take the absorbed form (decode steps and token trees)."""
        return types.SimpleNamespace(slot_map=slot_map, slots=slots, mask=None if causal else mask,
                                     parts=[latent_part(0, rows, seq_rows, cu_q, past, max_q, max_keys)])

    def ragged_batch(self, slot_map, meta, counts, past_lens):
        """Portions and decoded tokens, or token trees."""
        return types.SimpleNamespace(slot_map=slot_map, slots=meta.slots, mask=None if meta.causal else meta.mask_bits,
                                     parts=latent_parts(slot_map, meta, counts, past_lens, any(L.mix.expand for L in self.layers)))


def latent_part(r0, r1, seq_rows, cu_q, past, max_q, max_keys, expand=False, **kw):
    """A group of consecutive sequences of a batch: rows ``[r0, r1)``, ``cu_q`` counted from ``r0``."""
    return types.SimpleNamespace(r0=r0, r1=r1, seq_rows=seq_rows, cu_q=cu_q, past=past, max_q=max_q, max_keys=max_keys,
                                 seqs=int(seq_rows.numel()), expand=expand, **kw)


def latent_parts(slot_map, meta, counts, past_lens, may_expand: bool) -> list:
    """Sequence groups of a ragged batch in row order: short portions absorbed, and (where every sequence behind the first long
    portion is long too) the long ones expanded."""
    dev, B = slot_map.device, len(counts)
    k = B
    if meta.causal and may_expand:
        while k > 0 and counts[k - 1] >= EXPAND_MIN_TOKENS:
            k -= 1
    r_split = sum(counts[:k])
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)
    parts = []
    if k > 0:
        parts.append(latent_part(0, r_split, meta.seq_rows[:k], meta.cu_q[: k + 1], meta.past_lens[:k], max(counts[:k]),
                                 max(a + b for a, b in zip(counts[:k], past_lens[:k]))))
    if k < B:
        lens = [a + b for a, b in zip(counts[k:], past_lens[k:])]
        base = [sum(lens[:j]) for j in range(len(lens))]
        rows = meta.seq_rows[k:]
        key_slots = torch.cat([slot_map[rows[j].long(), :n] for j, n in enumerate(lens)])
        parts.append(latent_part(r_split, sum(counts), rows, (meta.cu_q[k:] - meta.cu_q[k]).contiguous(), meta.past_lens[k:],
                                 max(counts[k:]), max(lens), expand=True, keys=sum(lens), key_slots=key_slots,
                                 key_base=i32(base), key_map=torch.arange(sum(lens), dtype=torch.int32, device=dev).view(-1, 1)))
    return parts
