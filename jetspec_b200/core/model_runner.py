"""Single model-forward seam of the reference engine.

``ModelRunner.forward`` runs the decoder on a batch-1 token row against a
contiguous per-layer KV cache, optionally under a tree (ancestor) mask, and
returns logits plus the tapped hidden states the draft head conditions on.
Reference: ``jetspec/core/model_runner.py:90-154``.
"""
from __future__ import annotations

import math
from typing import Optional, Sequence

import torch

from ..ops import reference as ref


class DenseKVCache:
    """Contiguous ``(Hkv, capacity, D)`` K and V per layer with a shared length; a latent-attention model's latent rows
    are held as ``k`` with one head (and no ``v``).

    A recurrent layer holds the inputs of its recurrence as rows of the same kind (``rec``), which :meth:`crop` and
    :meth:`select` handle like K and V, and its state at an earlier position (``folded`` positions are in it).  The next
    forward first advances the state over the rows that are committed by then."""

    def __init__(self, cfg, device, dtype, capacity: int = 512):
        self.cfg, self.device, self.dtype = cfg, device, dtype
        self.length = 0
        self.capacity = 0
        self.k: list = []
        self.v: list = []
        self.rec: list = []
        self.folded = 0
        self.states = None
        if cfg.state_shapes() is not None:
            from ..runtime.state_pool import StatePool
            self.states = StatePool(cfg.state_shapes(), 1, device=device, dtype=dtype)
        self._grow(capacity)

    def _grow(self, cap: int) -> None:
        widths, shapes = self.cfg.latent_widths(), self.cfg.kv_shapes()
        if shapes is not None or widths is not None:
            rows = lambda heads, w: torch.zeros(heads, cap, w, dtype=self.dtype, device=self.device)
            shapes, widths = shapes or [None] * len(widths), widths or [None] * len(shapes)
            keys = lambda heads, dim, vdim, maps=1: rows(heads, dim * maps)
            nk = [keys(*s) if s is not None else rows(1, w) if w is not None else None for s, w in zip(shapes, widths)]
            nv = [rows(s[0], s[2]) if s is not None else None for s in shapes]
        else:
            L, Hkv, D = self.cfg.num_hidden_layers, self.cfg.num_key_value_heads, self.cfg.head_dim
            nk = [torch.zeros(Hkv, cap, D, dtype=self.dtype, device=self.device) for _ in range(L)]
            nv = [torch.zeros(Hkv, cap, D, dtype=self.dtype, device=self.device) for _ in range(L)]
        nr = []
        if self.states is not None:     # the inputs of each layer's recurrence, each as one head
            row = lambda w, f32: torch.zeros(1, cap, w, dtype=torch.float32 if f32 else self.dtype, device=self.device)
            nr = [tuple(row(*h) for h in c.held) if c is not None else () for c in self.states.shapes]
        for new, old in ((nk, self.k), (nv, self.v), ([x for r in nr for x in r], [x for r in self.rec for x in r])):
            for n, o in zip(new, old):
                if n is not None:
                    n[:, : self.length] = o[:, : self.length]
        self.k, self.v, self.rec, self.capacity = nk, nv, nr, cap

    def ensure(self, n: int) -> None:
        if n > self.capacity:
            self._grow(max(n, 2 * self.capacity))

    def get_seq_length(self) -> int:
        return self.length

    def crop(self, length: int) -> None:
        if self.folded > int(length):
            raise RuntimeError("a recurrent state cannot be cropped to an earlier position")
        self.length = min(self.length, int(length))

    def select(self, past_len: int, keep_tree_indices) -> None:
        """Keep the first ``past_len`` positions, then move the tree positions
        ``past_len + keep_tree_indices[i]`` directly behind them (in that order).

        This is the physical compaction of the accepted path
        (reference: ``_select_kv_cache``, ``jetspec/core/llm.py:86-112``).
        """
        n = len(keep_tree_indices)
        if (n and n <= 64 and self.v and self.cfg.kv_shapes() is None and self.cfg.latent_widths() is None and self.k[0].is_cuda and self.k[0].dtype == torch.bfloat16 and self.k[0].shape[-1] == 128
                and self.k[0].is_contiguous()):
            from ..ops import cuda_ext as X                   # compaction kernel (rows staged in shared memory)
            keep = torch.as_tensor(keep_tree_indices, dtype=torch.int32).to(self.device)
            for i in range(len(self.k)):
                X.kv_compact(self.k[i], self.v[i], past_len, keep)
            self.length = past_len + n
            return
        idx = torch.as_tensor(keep_tree_indices, dtype=torch.long, device=self.device) + past_len
        for t in (*self.k, *self.v, *(x for r in self.rec for x in r)):
            if t is not None:
                t[:, past_len:past_len + n] = t[:, idx]
        self.length = past_len + n

    def recur(self, layer: int, mixer, inputs, mask_bits):
        """Recurrence of a layer over new rows behind the cached ones.  The committed rows the state lacks are folded in
        first; the new rows are read out from it without being stored, as a tree (``mask_bits``, ``None``: a chain)."""
        past, T = self.length, inputs[0].shape[0]
        i32 = lambda *v: torch.tensor(v, dtype=torch.int32, device=self.device)
        state, conv = self.states.layer(layer)
        if past > self.folded:
            rows = [x[0, self.folded:past] for x in self.rec[layer]]
            mixer.mix(rows, state, conv, i32(0), i32(0, past - self.folded), i32(self.folded), None, True)
        for x, new in zip(self.rec[layer], inputs):
            x[0, past:past + T] = new
        if mask_bits is None:                          # on copies: the rows may yet be cropped
            state, conv = state[:1].clone(), conv[:1].clone() if conv is not None else None
        return mixer.mix(inputs, state, conv, i32(0), i32(0, T), i32(past), mask_bits, mask_bits is None)


class ModelRunner:
    def __init__(self, model):
        self.model = model
        self.cfg = model.config

    def _kernel_attention_ok(self, ids: torch.Tensor, T: int, ancestor) -> bool:
        cfg = self.cfg
        w = self.model.lm_head.weight
        if not hasattr(cfg, "head_dim"):
            return False
        if not (ids.is_cuda and w.dtype == torch.bfloat16 and cfg.head_dim == 128):
            return False
        if cfg.sliding_window and any(t == "sliding_attention" for t in (cfg.layer_types or [])):
            return False
        return ancestor is None or T <= 256

    @staticmethod
    def _kernel_attention_args(cache, past: int, T: int, ancestor, device) -> dict:
        """The contiguous cache seen as a one-sequence paged pool: slot ``i`` is position ``i``."""
        i32 = dict(dtype=torch.int32, device=device)
        cap = cache.k[0].shape[1]
        out = {"slot_map": torch.arange(cap, **i32).view(1, cap), "seq_rows": torch.zeros(1, **i32),
               "cu_q": torch.tensor([0, T], **i32), "past": torch.tensor([past], **i32),
               "mask_bits": None, "causal": ancestor is None}
        if ancestor is not None:
            from ..tree.ancestor import pack_ancestor_bits
            out["mask_bits"] = pack_ancestor_bits(ancestor.to(device))
        return out

    def new_cache(self, capacity: int = 512) -> DenseKVCache:
        p = self.model.lm_head.weight
        return DenseKVCache(self.cfg, p.device, p.dtype, capacity)

    @torch.inference_mode()
    def forward(self, input_ids: torch.Tensor, past_key_values: Optional[DenseKVCache] = None,
                position_ids: Optional[torch.Tensor] = None, output_hidden_states: bool = False,
                target_layer_ids: Optional[Sequence[int]] = None, ancestor: Optional[torch.Tensor] = None,
                last_position_logits_only: bool = False, attn_kernel: bool = False):
        """Forward ``input_ids (1, T)``; new K/V are appended at ``cache.length``.

        ``ancestor (T, T) bool`` switches the new-token block from causal to tree
        masking: key ``j`` of the block is visible to query ``i`` iff
        ``ancestor[i, j]``; the cached prefix is always visible (sliding-window
        layers additionally hide keys further than the window behind the query).
        ``attn_kernel`` runs attention on the tcgen05 tree-attention kernel over the contiguous cache (the
        counterpart of the reference's dense tree-attention kernel for this path,
        ``jetspec/core/tree_attention_kernel.py:63-216``) instead of the fp32 PyTorch formula; it applies on a CUDA
        device with bf16 weights, ``head_dim`` 128, no sliding-window layers and at most 256 tree nodes, and is
        ignored otherwise.
        Returns ``(logits (1, T or 1, V), cache, target_hidden (1, T, taps*H) or None)``.
        """
        cfg = self.cfg
        ids = input_ids.reshape(-1)
        T = ids.numel()
        cache = past_key_values if past_key_values is not None else self.new_cache(max(512, 2 * T))
        past = cache.length
        cache.ensure(past + T)
        pos = (position_ids.reshape(-1) if position_ids is not None
               else torch.arange(past, past + T, device=ids.device))
        vis = torch.ones(T, past + T, dtype=torch.bool, device=ids.device)
        vis[:, past:] = (ancestor.to(ids.device) if ancestor is not None
                         else torch.tril(torch.ones(T, T, dtype=torch.bool, device=ids.device)))
        key_pos = torch.cat((torch.arange(past, device=ids.device), pos))
        windows = {}
        use_kernel = bool(attn_kernel) and self._kernel_attention_ok(ids, T, ancestor)
        if use_kernel:
            kern = self._kernel_attention_args(cache, past, T, ancestor, ids.device)

        if hasattr(cfg, "head_dim"):
            Hq, Hkv, D = cfg.num_attention_heads, cfg.num_key_value_heads, cfg.head_dim
            g = Hq // Hkv
            scale = 1.0 / math.sqrt(D)

        def weights(s, seen, sink):
            """Softmax over the visible keys; ``sink``: learned numbers per head, or whether a key of score 0 takes part."""
            s = s.masked_fill(~seen, float("-inf"))
            if isinstance(sink, torch.Tensor):
                extra = sink.float().view(s.shape[:-2] + (1, 1)).expand(s.shape[:-1] + (1,))
            elif sink:
                extra = torch.zeros_like(s[..., :1])
            else:
                return torch.softmax(s, -1)
            return torch.softmax(torch.cat((s, extra), -1), -1)[..., :-1]

        def latent(layer: int, mixer, q, c):
            """Latent attention as the plain formula over the contiguous cache: keys and values are expanded."""
            cache.k[layer][0, past:past + T] = c
            rows, m = cache.k[layer][0, :past + T].float(), mixer.cfg
            C = rows[:, : m.kv_rank]
            K = (C @ mixer.k_up.weight.float().t()).view(past + T, m.heads, m.dim)
            V = (C @ mixer.v_up.weight.float().t()).view(past + T, m.heads, m.vdim)
            s = torch.einsum("nhd,lhd->hnl", q[..., : m.dim].float(), K)
            if m.rot_dim:
                s = s + torch.einsum("nhd,ld->hnl", q[..., m.dim:].float(), rows[:, m.kv_rank:])
            p = weights(s * m.scale, vis[None], mixer.sink)
            return torch.einsum("hnl,lhv->nhv", p, V).reshape(T, m.heads * m.vdim).to(q.dtype)

        def attn(layer: int, q, k, v):
            cache.k[layer][:, past:past + T] = k.transpose(0, 1)
            cache.v[layer][:, past:past + T] = v.transpose(0, 1)
            if use_kernel:
                from ..ops import cuda_ext as X
                return X.paged_tree_attention(q.view(T, Hq, D).contiguous(), cache.k[layer], cache.v[layer],
                                              kern["slot_map"], kern["seq_rows"], kern["cu_q"], kern["past"],
                                              kern["mask_bits"], scale, kern["causal"], T, max_keys=past + T)
            K = cache.k[layer][:, :past + T].float()
            V = cache.v[layer][:, :past + T].float()
            qf = q.float().view(T, Hkv, g, D)
            s = torch.einsum("nhgd,hld->hgnl", qf, K) * scale
            m = vis
            if cfg.sliding_window and cfg.layer_types[layer] == "sliding_attention":
                if "w" not in windows:
                    windows["w"] = vis & ((pos[:, None] - key_pos[None, :]) < cfg.sliding_window)
                m = windows["w"]
            s = s.masked_fill(~m[None, None], float("-inf"))
            p = torch.softmax(s, -1)
            return torch.einsum("hgnl,hld->nhgd", p, V).reshape(T, Hq * D).to(q.dtype)

        bits = None
        if ancestor is not None and cache.states is not None:
            from ..tree.ancestor import pack_ancestor_bits
            bits = pack_ancestor_bits(ancestor.to(ids.device))

        sources = cfg.kv_sources() if hasattr(cfg, "kv_sources") else None

        def window(layer: int, mixer, q, k, v):
            """Attention in a window, with pooled blocks or differential, as the plain formula over the contiguous cache.  A
            block's score is the mean of its tokens' scores, and its weight is shared out over their values."""
            m = mixer.cfg
            at = layer if sources is None else sources[layer]
            if k is not None:
                cache.k[at][:, past:past + T] = k.transpose(0, 1)
                cache.v[at][:, past:past + T] = v.transpose(0, 1)
            K, V = cache.k[at][:, :past + T].float(), cache.v[at][:, :past + T].float()
            seen = vis & ((pos[:, None] - key_pos[None, :] < m.window) | (key_pos < m.keep_first)[None]) if m.window else vis
            if m.pool:
                ends = (torch.arange(int(pos.max()) // m.pool + 1, device=ids.device) + 1) * m.pool - 1
                far = ends[None] <= pos[:, None] - m.window
                share = (key_pos[:, None] // m.pool == (ends // m.pool)[None]).float() / m.pool
            acc = []
            for i in range(m.maps):
                qi = q[:, i::m.maps].float().reshape(T, m.kv_heads, m.heads // m.kv_heads, m.dim)
                s = torch.einsum("nhgd,hld->hgnl", qi, K[..., i * m.dim:(i + 1) * m.dim]) * m.scale
                if m.pool:
                    all_s, both = torch.cat((s, (s * vis) @ share), -1), torch.cat((seen, far), -1)
                    p = weights(ref.softcapped(all_s, m.softcap), both[None, None], mixer.sink)
                    p = p[..., : past + T] + (p[..., past + T:] @ share.t()) * vis
                else:
                    p = weights(ref.softcapped(s, m.softcap), seen[None, None], mixer.sink)
                acc.append(torch.einsum("hgnl,hlv->nhgv", p, V).reshape(T, m.heads, m.vdim))
            o = acc[0] if m.diff is None else ref.differential(torch.stack(acc, 2), *mixer.differential())
            return o.reshape(T, m.heads * m.vdim).to(q.dtype)

        attn.latent, attn.window = latent, window
        attn.recur = lambda layer, mixer, *inputs: cache.recur(layer, mixer, inputs, bits)
        attn.delta = attn.recur
        taps = list(target_layer_ids) if (output_hidden_states or target_layer_ids is not None) and target_layer_ids else None
        rows = slice(T - 1, T) if last_position_logits_only else None
        logits, hidden = self.model(ids, pos, attn, tap_layers=taps, logits_rows=rows)
        if cache.states is not None:
            cache.folded = past
        cache.length = past + T
        return logits.unsqueeze(0), cache, (hidden.unsqueeze(0) if hidden is not None else None)
