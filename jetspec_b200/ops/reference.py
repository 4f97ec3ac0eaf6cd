"""Plain PyTorch implementations of every op the engine uses.

These run on any device and dtype and are the numerical oracle for the sm_100a
kernels (each kernel test compares against the function of the same name here,
evaluated in fp32).  They are also the only implementation used on CPU.

Shapes use T = number of token rows in the (ragged) batch, H = hidden size,
Hq/Hkv = query / key-value heads, D = head_dim, S = KV slots in the pool.
"""
from __future__ import annotations

import math
from typing import Optional

import torch
import torch.nn.functional as F


# --------------------------------------------------------------------------
# norms, rotary, activations
# --------------------------------------------------------------------------
def rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float = 1e-6) -> torch.Tensor:
    """Qwen3 RMSNorm over the last dim; fp32 math, result in ``x.dtype``."""
    xf = x.float()
    var = xf.pow(2).mean(-1, keepdim=True)
    return (xf * torch.rsqrt(var + eps) * weight.float()).to(x.dtype)


def add_rmsnorm(residual: torch.Tensor, x: torch.Tensor, weight: torch.Tensor, eps: float = 1e-6):
    """``residual += x`` then RMSNorm; returns ``(new_residual, normed)``."""
    r = (residual.float() + x.float()).to(residual.dtype)
    return r, rmsnorm(r, weight, eps)


def rope_inv_freq(head_dim: int, theta: float, device=None) -> torch.Tensor:
    idx = torch.arange(0, head_dim, 2, dtype=torch.float32, device=device)
    return 1.0 / (theta ** (idx / head_dim))


def rope_cos_sin(positions: torch.Tensor, head_dim: int, theta: float):
    """fp32 ``cos, sin`` of shape ``(T, D/2)`` for integer positions."""
    inv = rope_inv_freq(head_dim, theta, positions.device)
    ang = positions.to(torch.float32)[:, None] * inv[None, :]
    return ang.cos(), ang.sin()


def apply_rope(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor) -> torch.Tensor:
    """Rotate-half RoPE on ``x (T, heads, D)`` with ``cos/sin (T, D/2)``."""
    xf = x.float()
    half = xf.shape[-1] // 2
    x1, x2 = xf[..., :half], xf[..., half:]
    c, s = cos[:, None, :], sin[:, None, :]
    return torch.cat((x1 * c - x2 * s, x2 * c + x1 * s), dim=-1).to(x.dtype)


def silu_mul(gate_up: torch.Tensor) -> torch.Tensor:
    """SwiGLU on a fused ``[gate | up]`` row: ``silu(gate) * up``."""
    g, u = gate_up.float().chunk(2, dim=-1)
    return (F.silu(g) * u).to(gate_up.dtype)


def dynamic_tanh(x: torch.Tensor, alpha: torch.Tensor, weight: torch.Tensor, bias: torch.Tensor, out_dtype) -> torch.Tensor:
    """``tanh(alpha x) * weight + bias`` in fp32, result in ``out_dtype``."""
    return (torch.tanh(alpha.float() * x.float()) * weight.float() + bias.float()).to(out_dtype)


def gelu_tanh_mul(gate: torch.Tensor, up: torch.Tensor) -> torch.Tensor:
    """``gelu_tanh(gate) * up``, fp32 inside."""
    return (F.gelu(gate.float(), approximate="tanh") * up.float()).to(gate.dtype)


def relu_squared(x: torch.Tensor) -> torch.Tensor:
    r = torch.relu(x.float())
    return (r * r).to(x.dtype)


def linear(x: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``x (M, K) @ w (N, K)^T``; the weight layout of ``nn.Linear``."""
    return F.linear(x, w, bias)


def qkv_postprocess(qkv: torch.Tensor, q_norm_w: torch.Tensor, k_norm_w: torch.Tensor,
                    positions: torch.Tensor, num_q_heads: int, num_kv_heads: int, head_dim: int,
                    theta: float, eps: float):
    """Split a fused QKV row, per-head RMSNorm on q and k, then RoPE.

    Returns ``q (T, Hq, D)``, ``k (T, Hkv, D)``, ``v (T, Hkv, D)``.  The norm comes
    before the rotation, as in Qwen3 (reference: ``compiled_verify_stack.py:226-233``).
    """
    T = qkv.shape[0]
    qs, ks = num_q_heads * head_dim, num_kv_heads * head_dim
    q = qkv[:, :qs].reshape(T, num_q_heads, head_dim)
    k = qkv[:, qs:qs + ks].reshape(T, num_kv_heads, head_dim)
    v = qkv[:, qs + ks:].reshape(T, num_kv_heads, head_dim)
    q = rmsnorm(q, q_norm_w, eps)
    k = rmsnorm(k, k_norm_w, eps)
    cos, sin = rope_cos_sin(positions, head_dim, theta)
    return apply_rope(q, cos, sin), apply_rope(k, cos, sin), v.contiguous()


# --------------------------------------------------------------------------
# paged tree attention
# --------------------------------------------------------------------------
def pack_ancestor_bits(ancestor: torch.Tensor, words: int) -> torch.Tensor:
    """Pack a bool ``(n, n)`` ancestor matrix into ``(n, words)`` int32 bit rows.

    Bit ``j`` of row ``i`` is set when tree key ``j`` is visible to query ``i``.
    """
    n = ancestor.shape[0]
    out = torch.zeros(n, words, dtype=torch.int64, device=ancestor.device)
    a = ancestor.to(torch.int64)
    for w in range(min(words, (n + 31) // 32)):
        chunk = a[:, w * 32:(w + 1) * 32]
        sh = torch.arange(chunk.shape[1], device=a.device, dtype=torch.int64)
        out[:, w] = (chunk << sh).sum(-1)
    out = torch.where(out >= 2 ** 31, out - 2 ** 32, out)
    return out.to(torch.int32)


def unpack_ancestor_bits(bits: torch.Tensor, n: int) -> torch.Tensor:
    """Inverse of :func:`pack_ancestor_bits` for the first ``n`` columns."""
    b = bits.to(torch.int64) & 0xFFFFFFFF
    cols = torch.arange(n, device=bits.device)
    return ((b[:, cols // 32] >> (cols % 32)) & 1).bool()


def paged_tree_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor,
                         slot_map: torch.Tensor, seq_rows: torch.Tensor, cu_q: torch.Tensor,
                         past_lens: torch.Tensor, mask_bits: Optional[torch.Tensor],
                         scale: float, causal: bool = False) -> torch.Tensor:
    """Ragged multi-sequence attention over a slot-addressed KV pool.

    ``q (T, Hq, D)`` holds the query rows of all sequences back to back;
    sequence ``b`` owns rows ``cu_q[b]:cu_q[b+1]`` (n_b rows).  Its keys are the
    logical positions ``0 .. past_lens[b]+n_b-1`` whose KV rows live at
    ``k_pool[:, slot_map[seq_rows[b], pos]]``.  Every position below
    ``past_lens[b]`` is visible to every query; position ``past_lens[b]+j`` is
    visible to query ``i`` when bit ``j`` of ``mask_bits[cu_q[b]+i]`` is set, or,
    with ``causal=True``, when ``j <= i``.  ``k_pool/v_pool`` are ``(Hkv, S, D)``.
    Softmax is evaluated in fp32.  Returns ``(T, Hq*D)`` in ``q.dtype``.
    """
    T, Hq, D = q.shape
    Hkv = k_pool.shape[0]
    g = Hq // Hkv
    out = torch.empty(T, Hq * D, dtype=q.dtype, device=q.device)
    cu = cu_q.tolist()
    pl = past_lens.tolist()
    rows = seq_rows.tolist()
    for b in range(len(cu) - 1):
        s, e = cu[b], cu[b + 1]
        n = e - s
        if n == 0:
            continue
        past = pl[b]
        L = past + n
        slots = slot_map[rows[b], :L].long()
        k = k_pool[:, slots].float()  # (Hkv, L, D)
        v = v_pool[:, slots].float()
        qb = q[s:e].float().view(n, Hkv, g, D).permute(1, 2, 0, 3)  # (Hkv, g, n, D)
        scores = torch.einsum("hgnd,hld->hgnl", qb, k) * scale
        vis = torch.ones(n, L, dtype=torch.bool, device=q.device)
        if causal:
            vis[:, past:] = torch.tril(torch.ones(n, n, dtype=torch.bool, device=q.device))
        else:
            vis[:, past:] = unpack_ancestor_bits(mask_bits[s:e], n)
        scores = scores.masked_fill(~vis[None, None], float("-inf"))
        p = torch.softmax(scores, dim=-1)
        p = torch.nan_to_num(p, nan=0.0)  # a fully masked row yields zeros
        o = torch.einsum("hgnl,hld->hgnd", p, v)  # (Hkv, g, n, D)
        out[s:e] = o.permute(2, 0, 1, 3).reshape(n, Hq * D).to(q.dtype)
    return out


def latent_attention(q: torch.Tensor, w_uk: torch.Tensor, w_uv: torch.Tensor, pool: torch.Tensor,
                     slot_map: torch.Tensor, seq_rows: torch.Tensor, cu_q: torch.Tensor, past_lens: torch.Tensor,
                     mask_bits: Optional[torch.Tensor], scale: float, causal: bool = False,
                     sink: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Attention over slot-addressed latent rows, keys and values expanded from them.

    ``q (T, H, D + E)``; ``pool (S, >= R + E)`` holds one row ``c | e`` per slot; ``w_uk (H*D, R)`` and ``w_uv (H*V, R)`` give
    head ``h`` of a cached row the key ``w_uk[h] c | e`` and the value ``w_uv[h] c`` (``E`` may be 0).  Sequences, visibility
    and masks as in :func:`paged_tree_attention`; softmax in fp32, with ``sink (H,)`` its denominator also holds
    ``exp(sink)``.  Returns ``(T, H*V)`` in ``q.dtype``.
    """
    T, H, _ = q.shape
    R, D, V = w_uk.shape[1], w_uk.shape[0] // H, w_uv.shape[0] // H
    E = q.shape[2] - D
    wk, wv = w_uk.float().view(H, D, R), w_uv.float().view(H, V, R)
    out = torch.empty(T, H * V, dtype=q.dtype, device=q.device)
    cu, pl, rows = cu_q.tolist(), past_lens.tolist(), seq_rows.tolist()
    for b in range(len(cu) - 1):
        s, e = cu[b], cu[b + 1]
        n = e - s
        if n == 0:
            continue
        L = pl[b] + n
        row = pool[slot_map[rows[b], :L].long()].float()
        c, e_part = row[:, :R], row[:, R:R + E]
        k, v = torch.einsum("lr,hdr->hld", c, wk), torch.einsum("lr,hvr->hlv", c, wv)
        vis = torch.ones(n, L, dtype=torch.bool, device=q.device)
        vis[:, pl[b]:] = (torch.tril(torch.ones(n, n, dtype=torch.bool, device=q.device)) if causal
                          else unpack_ancestor_bits(mask_bits[s:e], n))
        sc = torch.einsum("nhd,hld->hnl", q[s:e, :, :D].float(), k)
        if E:
            sc = sc + torch.einsum("nhd,ld->hnl", q[s:e, :, D:].float(), e_part)
        sc = (sc * scale).masked_fill(~vis[None], float("-inf"))
        if sink is not None:
            sc = torch.cat((sc, sink.float().view(H, 1, 1).expand(H, n, 1)), -1)
        p = torch.nan_to_num(torch.softmax(sc, dim=-1), nan=0.0)[..., :L]
        out[s:e] = torch.einsum("hnl,hlv->nhv", p, v).reshape(n, H * V).to(q.dtype)
    return out


def latent_scatter(c: torch.Tensor, pool: torch.Tensor, slots: torch.Tensor) -> None:
    """Write ``c (T, R)`` into the first ``R`` columns of ``pool (S, >= R)`` at ``slots (T,)``."""
    pool[slots.long(), :c.shape[1]] = c.to(pool.dtype)


def kv_scatter(k: torch.Tensor, v: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor,
               slots: torch.Tensor) -> None:
    """Write ``k, v (T, Hkv, D)`` into ``(Hkv, S, D)`` pools at ``slots (T,)``."""
    idx = slots.long()
    k_pool[:, idx] = k.transpose(0, 1).to(k_pool.dtype)
    v_pool[:, idx] = v.transpose(0, 1).to(v_pool.dtype)


# --------------------------------------------------------------------------
# vocabulary heads
# --------------------------------------------------------------------------
def lm_head_argmax(h: torch.Tensor, w: torch.Tensor):
    """Greedy token per row without keeping the logits: ``(argmax (T,), max (T,))``."""
    logits = F.linear(h, w).float()
    val, idx = logits.max(dim=-1)
    return idx, val


def lm_head_topk_logprobs(h: torch.Tensor, w: torch.Tensor, k: int):
    """Per-row top-``k`` tokens and their full-vocabulary log-probabilities.

    Equivalent to ``topk(log_softmax(h @ w^T), k)``: the normaliser is over the
    whole vocabulary, which the cumulative-logprob tree ordering relies on
    (reference: ``jetspec/tree/_core/topk_build.py:10-15``).
    """
    logits = F.linear(h, w).float()
    lp = torch.log_softmax(logits, dim=-1)
    vals, idx = torch.topk(lp, k, dim=-1)
    return idx, vals


# --------------------------------------------------------------------------
# mixture of experts
# --------------------------------------------------------------------------
def moe_route(router_logits: torch.Tensor, top_k: int, renorm: bool):
    """fp32 softmax over experts, top-k, optional renormalisation of the kept mass."""
    probs = torch.softmax(router_logits.float(), dim=-1)
    w, idx = torch.topk(probs, top_k, dim=-1)
    if renorm:
        w = w / w.sum(-1, keepdim=True)
    return w, idx


def moe_forward(x: torch.Tensor, gate_w: torch.Tensor, w_gate_up: torch.Tensor, w_down: torch.Tensor,
                top_k: int, renorm: bool, router_logits: Optional[torch.Tensor] = None) -> torch.Tensor:
    """Sparse MoE block: route, run each expert's SwiGLU MLP on its tokens, combine.

    ``w_gate_up (E, 2I, H)`` and ``w_down (E, H, I)`` are the stacked expert weights
    in ``nn.Linear`` orientation.  Reference behaviour: ``jetspec/models/moe_fused.py:16-51``.
    """
    T, H = x.shape
    E = w_gate_up.shape[0]
    if router_logits is None:
        router_logits = F.linear(x, gate_w)
    wts, idx = moe_route(router_logits, top_k, renorm)
    out = torch.zeros(T, H, dtype=torch.float32, device=x.device)
    flat_e = idx.reshape(-1)
    flat_t = torch.arange(T, device=x.device).repeat_interleave(top_k)
    flat_w = wts.reshape(-1)
    for e in range(E):
        sel = (flat_e == e).nonzero(as_tuple=True)[0]
        if sel.numel() == 0:
            continue
        tok = flat_t[sel]
        h = F.linear(x[tok], w_gate_up[e])
        h = silu_mul(h)
        y = F.linear(h, w_down[e]).float()
        out.index_add_(0, tok, y * flat_w[sel, None])
    return out.to(x.dtype)


def sigmoid_route(logits: torch.Tensor, correction: torch.Tensor, top: int, scale: float):
    """fp32 scores ``s = sigmoid(logits)``; the ``top`` largest ``s + correction`` are chosen and weighted by
    ``s / (sum of the chosen s + 1e-20) * scale``.  Returns ``(weights, experts)``, largest choice score first."""
    s = torch.sigmoid(logits.float())
    idx = torch.topk(s + correction.float(), top, dim=-1).indices
    w = s.gather(-1, idx)
    return w / (w.sum(-1, keepdim=True) + 1e-20) * scale, idx


def sigmoid_moe(x: torch.Tensor, router_w: torch.Tensor, correction: torch.Tensor, w_up: torch.Tensor,
                w_down: torch.Tensor, top: int, scale: float) -> torch.Tensor:
    """Routed experts ``w_down[e] relu(w_up[e] x)^2`` with sigmoid routing; fp32 ``(T, H)``."""
    wts, idx = sigmoid_route(F.linear(x.float(), router_w.float()), correction, top, scale)
    return experts_relu_squared(x, wts, idx, w_up, w_down)


def experts_relu_squared(x, wts, idx, w_up, w_down) -> torch.Tensor:
    """``sum_j wts[:, j] * (w_down[idx_j] relu(w_up[idx_j] x)^2)``, summed in fp32."""
    out = torch.zeros(x.shape[0], w_down.shape[1], dtype=torch.float32, device=x.device)
    for e in idx.unique().tolist():
        tok, j = (idx == e).nonzero(as_tuple=True)
        y = F.linear(relu_squared(F.linear(x[tok], w_up[e])), w_down[e]).float()
        out.index_add_(0, tok, y * wts[tok, j].unsqueeze(-1))
    return out


# --------------------------------------------------------------------------
# sampling
# --------------------------------------------------------------------------
def sample(logits: torch.Tensor, temperature: float = 0.0, generator=None) -> torch.Tensor:
    """argmax when ``temperature < 1e-5``, else a draw from ``softmax(logits / T)``.

    Reference: ``jetspec/core/sampler.py:10-17``.
    """
    if temperature < 1e-5:
        return logits.argmax(dim=-1)
    probs = torch.softmax(logits.float() / temperature, dim=-1)
    flat = probs.reshape(-1, probs.shape[-1])
    return torch.multinomial(flat, 1, generator=generator).reshape(probs.shape[:-1])


# --------------------------------------------------------------------------
# window attention, gated delta rules, table-routed experts
# --------------------------------------------------------------------------
def rmsnorm_f32(x: torch.Tensor, weight: torch.Tensor, eps: float) -> torch.Tensor:
    """RMS norm of fp32 rows, fp32 result."""
    x = x.float()
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * weight.float()


def linear_f32(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """``x @ w.T`` with the product left in fp32."""
    return F.linear(x.float(), w.float())


def pair_freq(dims: int, base: float, device=None) -> torch.Tensor:
    """``base^(-2i/dims)`` for the ``dims // 2`` rotated pairs, evaluated in double and rounded to fp32 once."""
    return torch.tensor([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=torch.float32, device=device)


def rotate_norm(x: torch.Tensor, positions: torch.Tensor, dims: int, base: float, eps: Optional[float]) -> torch.Tensor:
    """Rotate the pairs ``(2i, 2i+1)`` of the first ``dims`` entries of every head of ``x (T, heads, D)``; with ``eps``
    every head is then divided by its root mean square.  fp32 math, result in ``x.dtype``."""
    y = x.float().clone()
    n = dims // 2
    if n:
        a = positions.to(torch.float32)[:, None] * pair_freq(dims, base, x.device)[None]
        c, s = a.cos()[:, None], a.sin()[:, None]
        u, v = y[..., 0:2 * n:2].clone(), y[..., 1:2 * n:2].clone()
        y[..., 0:2 * n:2], y[..., 1:2 * n:2] = u * c - v * s, v * c + u * s
    if eps is not None:
        y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps)
    return y.to(x.dtype)


def window_scatter(k: torch.Tensor, v: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, slots: torch.Tensor, maps: int = 1) -> None:
    """:func:`kv_scatter` into pools whose rows may be wider than the heads; a key of several ``maps`` has an equal share of the
    row for each."""
    if maps > 1:
        wide = k.new_zeros(*k.shape[:2], maps, k_pool.shape[-1] // maps)
        wide[..., : k.shape[-1] // maps] = k.view(*k.shape[:2], maps, -1)
        k = wide.flatten(2)
    kv_scatter(k, v, k_pool[..., : k.shape[-1]], v_pool[..., : v.shape[-1]], slots)


def pool_blocks(k_pool: torch.Tensor, v_pool: torch.Tensor, kb_pool: torch.Tensor, vb_pool: torch.Tensor, block_map: torch.Tensor, P: int,
                slot_map: torch.Tensor, seq_rows: torch.Tensor, cu_q: torch.Tensor, past_lens: torch.Tensor) -> None:
    """Pool the blocks of ``P`` tokens whose last token is among the sequences' new rows: their rows ``block_map[row, b]`` of
    ``kb_pool`` and ``vb_pool`` get the means of the cached keys and values."""
    cu, pl, rows = cu_q.tolist(), past_lens.tolist(), seq_rows.tolist()
    for i in range(len(cu) - 1):
        first, stop = pl[i] // P, (pl[i] + cu[i + 1] - cu[i]) // P
        if stop > first:
            slots, at = slot_map[rows[i], first * P:stop * P].long(), block_map[rows[i], first:stop].long()
            for src, dst in ((k_pool, kb_pool), (v_pool, vb_pool)):
                dst[:, at] = src[:, slots].float().view(src.shape[0], stop - first, P, -1).mean(2).to(dst.dtype)


def softcapped(s: torch.Tensor, cap: float) -> torch.Tensor:
    return cap * torch.tanh(s / cap) if cap > 0 else s


def differential(a: torch.Tensor, lam: torch.Tensor, share: float, eps: float) -> torch.Tensor:
    """Outputs ``a (T, H, 2, V)`` of a head's two maps to ``share * rms_norm(a1 - lam a2)``, fp32 ``(T, H, V)``."""
    o = a[:, :, 0].float() - lam.float() * a[:, :, 1].float()
    return share * o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + eps)


def window_attention(q: torch.Tensor, k_pool: torch.Tensor, v_pool: torch.Tensor, vdim: int, slot_map: torch.Tensor,
                     seq_rows: torch.Tensor, cu_q: torch.Tensor, past_lens: torch.Tensor, mask_bits: Optional[torch.Tensor],
                     scale: float, window: int, sink, causal: bool = False, keep_first: int = 0, softcap: float = 0.0,
                     blocks=None, diff=None) -> torch.Tensor:
    """:func:`paged_tree_attention` with a window, an optional sink, and heads narrower than the pools' rows.  ``sink``: whether
    a valueless key of score 0 takes part in the softmax, or such a key's score per head ``(Hq,)``.  A row sees the last
    ``window`` tokens of its own path (itself included; 0: all of them) and those at positions below ``keep_first``: in a tree a
    node's position is the committed length plus its number of proper ancestors.  ``softcap``: see :func:`softcapped`.

    ``blocks = (kb_pool, vb_pool, block_map, P)``: a row also sees, in the same softmax, one pooled key and value for each block
    of ``P`` positions that ends before its window.  Blocks that end in committed tokens or in a portion are read from their
    rows; those that reach into a token tree are the means over the row's own path.

    ``diff = (lam, share, eps)``: ``q (T, 2 Hq, D)`` holds two vectors a head and the pools' rows two keys, whose attentions over
    the same values are combined by :func:`differential`.  Returns ``(T, Hq*vdim)``."""
    T, Hq, D = q.shape
    Hkv, maps = k_pool.shape[0], 1 if diff is None else 2
    Hq //= maps
    g, km = Hq // Hkv, k_pool.shape[2] // maps
    out = torch.empty(T, Hq * vdim, dtype=q.dtype, device=q.device)
    cu, pl, rows = cu_q.tolist(), past_lens.tolist(), seq_rows.tolist()
    for b in range(len(cu) - 1):
        s, e = cu[b], cu[b + 1]
        n, past = e - s, pl[b]
        if n == 0:
            continue
        slots = slot_map[rows[b], :past + n].long()
        anc = (torch.tril(torch.ones(n, n, dtype=torch.bool, device=q.device)) if causal else unpack_ancestor_bits(mask_bits[s:e], n))
        pos = past + anc.sum(-1) - 1
        key_pos = torch.cat((torch.arange(past, device=q.device), pos))
        path = torch.cat((torch.ones(n, past, dtype=torch.bool, device=q.device), anc), -1)
        vis = path
        if window > 0:
            vis = path & ((pos[:, None] - key_pos[None] < window) | (key_pos < keep_first)[None])
        stored = 0
        if blocks is not None:
            kb_pool, vb_pool, block_map, P = blocks
            stored = (past + n if causal else past) // P
            at = block_map[rows[b], :stored].long()
            ends = (torch.arange(max(stored, int(pos.max()) // P + 1), device=q.device) + 1) * P - 1
            far = ends[None] <= pos[:, None] - window
            # blocks that reach into the tree: shares of the row's path tokens
            share = torch.zeros(past + n, far.shape[1], device=q.device)
            share[torch.arange(past + n, device=q.device), (key_pos // P).clamp(max=far.shape[1] - 1)] = 1.0 / P
        acc = []
        for m in range(maps):
            k, v = k_pool[:, slots, m * km:m * km + D].float(), v_pool[:, slots, :vdim].float()
            qm = q[s:e, m::maps].float().reshape(n, Hkv, g, D)
            raw = torch.einsum("nhgd,hld->hgnl", qm, k) * scale
            sc = softcapped(raw, softcap).masked_fill(~vis, float("-inf"))
            if blocks is not None:
                kb, vb = kb_pool[:, at, :D].float(), vb_pool[:, at, :vdim].float()
                sb = torch.cat((torch.einsum("nhgd,hld->hgnl", qm, kb) * scale, (raw * path) @ share[:, stored:]), -1)
                sc = torch.cat((sc, softcapped(sb, softcap).masked_fill(~far, float("-inf"))), -1)
            if isinstance(sink, torch.Tensor):
                sc = torch.cat((sc, sink.float().view(Hkv, g, 1, 1).expand(Hkv, g, n, 1)), -1)
            elif sink:
                sc = torch.cat((sc, torch.zeros_like(sc[..., :1])), -1)
            p = torch.nan_to_num(torch.softmax(sc, dim=-1), nan=0.0)
            w = p[..., : past + n]
            if blocks is not None:
                pb = p[..., past + n:past + n + far.shape[1]]
                w = w + (pb[..., stored:] @ share[:, stored:].t()) * path
            o = torch.einsum("hgnl,hlv->nhgv", w, v)
            if blocks is not None:
                o = o + torch.einsum("hgnl,hlv->nhgv", pb[..., :stored], vb)
            acc.append(o.reshape(n, Hq, vdim))
        o = acc[0] if diff is None else differential(torch.stack(acc, 2), *diff)
        out[s:e] = o.reshape(n, Hq * vdim).to(q.dtype)
    return out


def delta_inputs(y: torch.Tensor, taps: torch.Tensor, z: torch.Tensor, b: torch.Tensor, A_log: torch.Tensor,
                 dt_bias: torch.Tensor, cfg):
    """One token's delta-rule inputs from its window ``y (taps, channels)`` of un-convolved rows (oldest first), decay
    inputs ``z`` and step-size inputs ``b``: ``q, k (H, D)``, ``v (H, V)``, ``g (H, D or 1)``, ``beta (H,)``, fp32."""
    H, G, D, V = cfg.heads, cfg.kv_heads, cfg.dim, cfg.vdim
    c = F.silu((y.float() * taps.float().t()).sum(0))
    q, k, v = c[: G * D].view(G, D), c[G * D: 2 * G * D].view(G, D), c[2 * G * D:].view(H, V)
    unit = lambda x: x / torch.sqrt(x.pow(2).sum(-1, keepdim=True) + 1e-6)
    q, k = (unit(x).repeat_interleave(H // G, 0) for x in (q, k))
    g = torch.exp(-torch.exp(A_log.float())[:, None] * F.softplus(z.float() + dt_bias.float()).view(H, -1))
    return q * D ** -0.5, k, v, g, torch.sigmoid(b.float())


def delta_mix(pre: torch.Tensor, z: torch.Tensor, b: torch.Tensor, taps: torch.Tensor, A_log: torch.Tensor,
              dt_bias: torch.Tensor, cfg, state: torch.Tensor, conv: torch.Tensor, rows: torch.Tensor, cu_q: torch.Tensor,
              past_lens: torch.Tensor, mask_bits: Optional[torch.Tensor], causal: bool = True) -> torch.Tensor:
    """Short convolutions and the gated delta rule over a ragged batch.

    ``pre (T, channels)`` are un-convolved q | k | v rows; sequence ``i`` owns rows ``cu_q[i]:cu_q[i+1]``, its state is
    ``state[rows[i]] (H, D, V)`` and its last convolution inputs the ring ``conv[rows[i]] (taps, channels)``, the row of
    position ``p`` in entry ``p % taps``.  A sequence whose ``past_lens`` is 0 starts from zeros whatever its slot holds.  Causal: tokens follow one another and
    the states advance.  With ``mask_bits`` (a token tree, parents before children) every node continues its parent's
    state and the stored states stay as they are.  Per head ``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q``.
    Returns the read-outs, fp32 ``(T, H, V)``."""
    n_old = taps.shape[1] - 1
    out = torch.empty(pre.shape[0], cfg.heads, cfg.vdim, dtype=torch.float32, device=pre.device)
    cu, pl, rl = cu_q.tolist(), past_lens.tolist(), rows.tolist()
    for i in range(len(cu) - 1):
        s, e, row = cu[i], cu[i + 1], rl[i]
        n = e - s
        if n == 0:
            continue
        past, S0 = pl[i], state[row].clone()
        if past == 0:
            S0 = torch.zeros_like(S0)
        y0 = torch.zeros(n_old, pre.shape[1], dtype=pre.dtype, device=pre.device)
        for m in range(1, min(n_old, past) + 1):
            y0[n_old - m] = conv[row, (past - m) % taps.shape[1]]
        anc = None if causal else unpack_ancestor_bits(mask_bits[s:e], n).cpu()
        kept = []                                       # per row: state behind it, un-convolved rows up to it
        for t in range(n):
            if causal:
                parent = t - 1
            else:
                up = [j for j in range(t) if bool(anc[t, j])]
                parent = up[-1] if up else -1
            S, y = kept[parent] if parent >= 0 else (S0, y0)
            y = torch.cat((y, pre[s + t: s + t + 1]), 0)
            q, k, v, g, beta = delta_inputs(y[-(n_old + 1):], taps, z[s + t], b[s + t], A_log, dt_bias, cfg)
            S = S * g[..., None]
            u = beta[:, None] * (v - torch.einsum("hdv,hd->hv", S, k))
            S = S + k[..., None] * u[:, None]
            out[s + t] = torch.einsum("hdv,hd->hv", S, q)
            kept.append((S, y[1:] if n_old else y[:0]))
            if causal and t:
                kept[t - 1] = None
        if causal:
            state[row] = kept[-1][0]
            for t in range(max(0, n - n_old), n):
                conv[row, (past + t) % taps.shape[1]] = pre[s + t].to(conv.dtype)
    return out


def gated_head_norm(o: torch.Tensor, weight: Optional[torch.Tensor], gate: torch.Tensor, kind: str, eps: float) -> torch.Tensor:
    """``o (T, H, V)`` divided by its root mean square per head, times ``weight (V,)`` if any, times ``silu`` or ``sigmoid``
    of ``gate (T, H*V)``; fp32 math, result in ``gate.dtype``."""
    y = o.float() / torch.sqrt(o.float().pow(2).mean(-1, keepdim=True) + eps)
    if weight is not None:
        y = y * weight.float()
    a = F.silu(gate.float()) if kind == "silu" else torch.sigmoid(gate.float())
    return (y.reshape(gate.shape) * a).to(gate.dtype)


def experts_swiglu(x, idx, w_gate, w_up, w_down) -> torch.Tensor:
    """Mean over the token's experts ``idx (T, top)`` of ``w_down[e] (silu(w_gate[e] x) * w_up[e] x)``, fp32 sums."""
    out = torch.zeros(x.shape[0], w_down.shape[1], dtype=torch.float32, device=x.device)
    for e in idx.unique().tolist():
        tok = (idx == e).nonzero(as_tuple=True)[0]
        a = silu_mul(torch.cat((F.linear(x[tok], w_gate[e]), F.linear(x[tok], w_up[e])), -1))
        out.index_add_(0, tok, F.linear(a, w_down[e]).float())
    return out / idx.shape[1]


# --------------------------------------------------------------------------
# general rotations, gates per head, retention
# --------------------------------------------------------------------------
def xielu(x: torch.Tensor, up: float, down: float) -> torch.Tensor:
    """``up x^2 + x / 2`` for positive ``x``, ``down (e^x - 1 - x) + x / 2`` below; 32-bit math."""
    z = x.float()
    return (torch.where(z > 0, up * z * z, down * (torch.expm1(z.clamp(max=0.0)) - z)) + 0.5 * z).to(x.dtype)


def query_temperature(x: torch.Tensor, positions: torch.Tensor, every: int, coef: float) -> torch.Tensor:
    """``x (T, ...)`` times ``1 + coef ln(floor((p + 1) / every) + 1)`` of each row's position ``p``."""
    f = 1.0 + coef * torch.log(((positions + 1) // every + 1).float())
    return (x.float() * f.view(-1, *[1] * (x.dim() - 1))).to(x.dtype)


def depth_average(history: list, weights: torch.Tensor) -> torch.Tensor:
    """``sum_j weights[j] history[j]`` of fp32 rows."""
    w = weights.float()
    out = history[0] * w[0]
    for j in range(1, len(history)):
        out = out + history[j] * w[j]
    return out


def gelu_erf(x: torch.Tensor) -> torch.Tensor:
    """Exact gelu, fp32 inside."""
    return F.gelu(x.float()).to(x.dtype)


def rotate(x: torch.Tensor, positions: torch.Tensor, rot, out_dtype: Optional[torch.dtype] = None) -> torch.Tensor:
    """Rotate the pairs ``rot`` (a ``RotaryConfig``) names in every head of ``x (T, heads, D)``; the entries behind
    ``rot.dims`` pass unchanged.  fp32 math."""
    y, n = x.float().clone(), rot.dims // 2
    if n:
        f = torch.tensor(rot.frequencies(), dtype=torch.float32, device=x.device)
        a, amp = positions.to(torch.float32)[:, None] * f, rot.amplitude()
        c, s = (amp * a.cos())[:, None], (amp * a.sin())[:, None]
        first, second = (slice(0, n), slice(n, 2 * n)) if rot.pairing == "half" else (slice(0, 2 * n, 2), slice(1, 2 * n, 2))
        u, v = y[..., first].clone(), y[..., second].clone()
        y[..., first], y[..., second] = u * c - v * s, v * c + u * s
    return y.to(out_dtype or x.dtype)


def head_gate(y: torch.Tensor, logits: torch.Tensor) -> torch.Tensor:
    """``y (T, H*V)`` with head ``h``'s columns times ``sigmoid(logits[:, h])``, ``logits (T, H)``."""
    T, H = logits.shape
    return (y.float().view(T, H, -1) * torch.sigmoid(logits.float())[..., None]).reshape(T, -1).to(y.dtype)


def retention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cfg, state: torch.Tensor, rows: torch.Tensor, cu_q: torch.Tensor,
              past_lens: torch.Tensor, mask_bits: Optional[torch.Tensor], causal: bool = True) -> torch.Tensor:
    """Linear attention with one fixed decay per head over a ragged batch: ``S <- decay S + k v^T; o = S^T q``.

    ``q, k (T, H*D)`` and ``v (T, H*V)`` rows, ``state (slots, H, D, V)`` fp32; sequences, fresh starts and trees as in
    :func:`delta_mix`.  Returns the read-outs, fp32 ``(T, H, V)``."""
    H, D, V = cfg.heads, cfg.dim, cfg.vdim
    T = q.shape[0]
    q, k, v = q.float().view(T, H, D), k.float().view(T, H, D), v.float().view(T, H, V)
    decay = torch.tensor(cfg.decay, dtype=torch.float32, device=q.device)[:, None, None]
    out = torch.empty(T, H, V, dtype=torch.float32, device=q.device)
    cu, pl, rl = cu_q.tolist(), past_lens.tolist(), rows.tolist()
    for i in range(len(cu) - 1):
        s, e = cu[i], cu[i + 1]
        S0 = state[rl[i]].clone() if pl[i] > 0 else torch.zeros_like(state[rl[i]])
        anc = None if causal else unpack_ancestor_bits(mask_bits[s:e], e - s).cpu()
        kept = []
        for t in range(s, e):
            if causal:
                parent = len(kept) - 1
            else:
                up = [j for j in range(t - s) if bool(anc[t - s, j])]
                parent = up[-1] if up else -1
            S = decay * (kept[parent] if parent >= 0 else S0) + k[t][..., None] * v[t][:, None]
            out[t] = torch.einsum("hdv,hd->hv", S, q[t])
            if causal and kept:
                kept[-1] = None
            kept.append(S)
        if causal and kept:
            state[rl[i]] = kept[-1]
    return out
