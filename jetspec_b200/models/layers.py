"""Building blocks that are not Qwen3's: Dynamic Tanh, latent attention, GELU and xIELU MLPs, sigmoid-routed experts; attention
in a window, with sinks, with pooled blocks or differential, gated delta rules, retention, two mixers side by side, table-routed
experts.

Each takes its sizes and constants as arguments, so a design can combine them freely; the Qwen3 twins (RMSNorm, grouped
query attention, SwiGLU MLP, softmax-routed experts) are in :mod:`jetspec_b200.models.qwen3`.  ``forward`` is the
unfused form on :mod:`jetspec_b200.ops`, in any dtype and on any device; the fused kernel forms of whole decoders made
of these blocks are :mod:`jetspec_b200.engine.latent_stack`, :mod:`jetspec_b200.engine.hybrid_stack` and
:mod:`jetspec_b200.engine.prenorm_stack`.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from .config import (DeltaConfig, LatentAttentionConfig, RetentionConfig, RoutedExpertsConfig, TableExpertsConfig,
                     WindowAttentionConfig)


class DynamicTanh(nn.Module):
    """``tanh(alpha x) * weight + bias``: a norm without statistics.  32-bit math, output in ``out_dtype``."""

    def __init__(self, dim: int):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(dim))
        self.bias = nn.Parameter(torch.zeros(dim))
        self.alpha = nn.Parameter(torch.tensor(0.5))

    def forward(self, x, out_dtype=None):
        return ops.dynamic_tanh(x, self.alpha, self.weight, self.bias, out_dtype or self.weight.dtype)


class LatentAttention(nn.Module):
    """Attention whose keys and values (and, with a ``q_rank``, queries) pass through RMS-normed latents; only the K/V latent
    is cached, with the rotated key part all heads share where the design has one.

    ``forward(h, attend, positions)``: ``attend(q, c)`` stores the new cache rows ``c (T, kv_rank + rot_dim)`` and returns the
    attention of ``q (T, heads, dim + rot_dim)`` over the cached rows, ``(T, heads * vdim)``."""

    def __init__(self, cfg: LatentAttentionConfig, hidden: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        lin = lambda i, o: nn.Linear(i, o, bias=False)
        qd = cfg.heads * (cfg.dim + cfg.rot_dim)
        if cfg.q_rank:
            self.q_down, self.q_up = lin(hidden, cfg.q_rank), lin(cfg.q_rank, qd)
            self.q_norm = nn.Parameter(torch.ones(cfg.q_rank))
        else:
            self.q_proj = lin(hidden, qd)
        self.kv_down = lin(hidden, cfg.row)
        self.k_up, self.v_up = lin(cfg.kv_rank, cfg.heads * cfg.dim), lin(cfg.kv_rank, cfg.heads * cfg.vdim)
        self.o_proj = lin(cfg.heads * cfg.vdim, hidden)
        self.kv_norm = nn.Parameter(torch.ones(cfg.kv_rank))
        self.sink = nn.Parameter(torch.zeros(cfg.heads)) if cfg.sink_logits else None
        if cfg.gate:
            self.gate_proj = lin(hidden, cfg.heads)

    def forward(self, h, attend, positions=None):
        m, T = self.cfg, h.shape[0]
        if m.q_rank:
            q = ops.linear(ops.rmsnorm(ops.linear(h, self.q_down.weight), self.q_norm, self.eps), self.q_up.weight)
        else:
            q = ops.linear(h, self.q_proj.weight)
        q, c = q.view(T, m.heads, m.dim + m.rot_dim), ops.linear(h, self.kv_down.weight)
        if m.rot is None:
            c = ops.rmsnorm(c, self.kv_norm, self.eps)
        else:
            q = torch.cat((q[..., : m.dim], ops.rotate(q[..., m.dim:], positions, m.rot)), -1)
            shared = ops.rotate(c[:, None, m.kv_rank:], positions, m.rot)[:, 0]
            c = torch.cat((ops.rmsnorm(c[:, : m.kv_rank].contiguous(), self.kv_norm, self.eps), shared), -1)
        y = attend(q, c)
        if m.gate:
            y = ops.head_gate(y, ops.linear_f32(h, self.gate_proj.weight))
        return ops.linear(y, self.o_proj.weight)


class GeluMLP(nn.Module):
    """``down(gelu_tanh(gate(h)) * up(h))``."""

    def __init__(self, hidden: int, inter: int):
        super().__init__()
        self.gate_proj = nn.Linear(hidden, inter, bias=False)
        self.up_proj = nn.Linear(hidden, inter, bias=False)
        self.down_proj = nn.Linear(inter, hidden, bias=False)

    def forward(self, h):
        a = ops.gelu_tanh_mul(ops.linear(h, self.gate_proj.weight), ops.linear(h, self.up_proj.weight))
        return ops.linear(a, self.down_proj.weight)


class GeluErfMLP(nn.Module):
    """``down(gelu(up(h)))`` with the exact (erf) gelu."""

    def __init__(self, hidden: int, inter: int):
        super().__init__()
        self.up_proj = nn.Linear(hidden, inter, bias=False)
        self.down_proj = nn.Linear(inter, hidden, bias=False)

    def forward(self, h):
        return ops.linear(ops.gelu_erf(ops.linear(h, self.up_proj.weight)), self.down_proj.weight)


class XieluMLP(nn.Module):
    """``down(xielu(up(h)))``; the activation's two learned numbers ``act`` pass through a softplus."""

    def __init__(self, hidden: int, inter: int):
        super().__init__()
        self.up_proj = nn.Linear(hidden, inter, bias=False)
        self.down_proj = nn.Linear(inter, hidden, bias=False)
        self.act = nn.Parameter(torch.zeros(2))
        self._coef = None

    def coefficients(self) -> tuple:
        """Factors of the quadratic and of the exponential part, as host numbers (read once per parameter value)."""
        key = (self.act.data_ptr(), self.act._version)
        if self._coef is None or self._coef[0] != key:
            up, down = torch.nn.functional.softplus(self.act.detach().double().cpu()).tolist()
            self._coef = (key, (up, 0.5 + down))
        return self._coef[1]

    def forward(self, h):
        return ops.linear(ops.xielu(ops.linear(h, self.up_proj.weight), *self.coefficients()), self.down_proj.weight)


class SigmoidMoE(nn.Module):
    """Experts chosen by ``sigmoid(router(h)) + correction`` and weighted by the normalised sigmoid without it; expert =
    ``down(relu(up(h))^2)``.  A shared expert of the same form, gated by ``sigmoid(shared_gate(h))``, is added."""

    def __init__(self, cfg: RoutedExpertsConfig, hidden: int):
        super().__init__()
        self.cfg = cfg
        self.router = nn.Linear(hidden, cfg.experts, bias=False)
        self.correction = nn.Parameter(torch.zeros(cfg.experts))
        self.w_up = nn.Parameter(torch.empty(cfg.experts, cfg.ff, hidden))
        self.w_down = nn.Parameter(torch.empty(cfg.experts, hidden, cfg.ff))
        if cfg.shared_ff:
            self.shared_up = nn.Linear(hidden, cfg.shared_ff, bias=False)
            self.shared_down = nn.Linear(cfg.shared_ff, hidden, bias=False)
            self.shared_gate = nn.Linear(hidden, 1, bias=False)

    def forward(self, h):
        c = self.cfg
        y = ops.sigmoid_moe(h, self.router.weight, self.correction, self.w_up, self.w_down, c.top, c.scale)
        if c.shared_ff:
            s = ops.linear(ops.relu_squared(ops.linear(h, self.shared_up.weight)), self.shared_down.weight)
            gate = torch.sigmoid(h.float() @ self.shared_gate.weight.float().t())
            y = y + gate * s.float()
        return y


class PlainRMSNorm(nn.Module):
    """RMS norm of fp32 rows; 32-bit math and output."""

    def __init__(self, dim: int, eps: float):
        super().__init__()
        self.eps = eps
        self.weight = nn.Parameter(torch.ones(dim))

    def scale(self):
        """What the normed rows are multiplied by, fp32."""
        return self.weight.float()

    def forward(self, x):
        return ops.rmsnorm_f32(x, self.weight, self.eps)


class OffsetRMSNorm(PlainRMSNorm):
    """:class:`PlainRMSNorm` whose weight is stored as its distance from one."""

    def __init__(self, dim: int, eps: float):
        super().__init__(dim, eps)
        nn.init.zeros_(self.weight)

    def scale(self):
        return self.weight.float() + 1.0

    def forward(self, x):
        return ops.rmsnorm_f32(x, self.scale(), self.eps)


class WindowAttention(nn.Module):
    """Attention over grouped K/V heads, in a sliding window or over the whole past.  Options (see the configuration): rotation
    in neighbouring or half pairs, norm of q and k per head behind it or over the whole projections ahead of it, kept first
    tokens, pooled blocks behind the window, a valueless sink of score 0 or a learned one per head, capped scores, two
    attention maps a head whose difference counts, a temperature that grows with the position, values that are the keys,
    keys and values of another layer, a sigmoid gate per head, biases.

    ``forward(h, positions, attend)``: ``attend(q, k, v)`` stores the new K/V rows (``None`` for both: there are none) and
    returns the attention, ``(T, heads * vdim)``."""

    def __init__(self, cfg: WindowAttentionConfig, hidden: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        lin = lambda i, o: nn.Linear(i, o, bias=cfg.bias)
        self.q_proj = lin(hidden, cfg.heads * cfg.maps * cfg.dim)
        self.k_proj = lin(hidden, cfg.kv_heads * cfg.maps * cfg.dim) if cfg.kv_from is None else None
        self.v_proj = lin(hidden, cfg.kv_heads * cfg.vdim) if cfg.kv_from is None and not cfg.tie_values else None
        self.o_proj = nn.Linear(cfg.heads * cfg.vdim, hidden, bias=cfg.bias if cfg.o_bias is None else cfg.o_bias)
        if cfg.proj_norm:
            self.q_norm, self.k_norm = nn.Parameter(torch.ones(cfg.heads * cfg.dim)), nn.Parameter(torch.ones(cfg.kv_heads * cfg.dim))
        self.sink_logits = nn.Parameter(torch.zeros(cfg.heads)) if cfg.sink_logits else None
        if cfg.gate:
            self.gate_proj = nn.Linear(hidden, cfg.heads, bias=False)
        if cfg.diff is not None:
            self.lq1, self.lk1, self.lq2, self.lk2 = (nn.Parameter(torch.zeros(cfg.dim)) for _ in range(4))

    def differential(self):
        """``(lambda, share, eps)`` of :func:`ops.reference.differential`; ``None`` with one map a head."""
        if self.cfg.diff is None:
            return None
        dot = lambda a, b: torch.exp((a.float() * b.float()).sum())
        return dot(self.lq1, self.lk1) - dot(self.lq2, self.lk2) + self.cfg.diff, 1.0 - self.cfg.diff, self.eps

    @property
    def sink(self):
        """What the attention ops take: learned numbers per head, or whether a sink of score 0 takes part."""
        return self.sink_logits if self.sink_logits is not None else self.cfg.sink

    def forward(self, h, positions, attend):
        c, T = self.cfg, h.shape[0]
        q, k, v = (ops.linear(h, p.weight, p.bias) if p is not None else None for p in (self.q_proj, self.k_proj, self.v_proj))
        if c.tie_values:
            v = k
        if c.proj_norm:
            q, k = ops.rmsnorm(q, self.q_norm, self.eps), ops.rmsnorm(k, self.k_norm, self.eps)

        def turn(x, heads):
            x = x.view(T, heads, c.dim)
            if c.rot is not None:
                return ops.rotate(x, positions, c.rot)
            return ops.rotate_norm(x, positions, c.rot_dims, c.rot_base, self.eps if c.qk_norm else None)
        q = turn(q, c.heads * c.maps)
        if c.temp_every:
            q = ops.query_temperature(q, positions, c.temp_every, c.temp_coef)
        if k is not None:
            k, v = turn(k, c.kv_heads * c.maps).reshape(T, c.kv_heads, c.maps * c.dim), v.view(T, c.kv_heads, c.vdim)
        y = attend(q, k, v)
        if c.gate:
            y = ops.head_gate(y, ops.linear_f32(h, self.gate_proj.weight))
        return ops.linear(y, self.o_proj.weight, self.o_proj.bias)


class GatedDelta(nn.Module):
    """Gated delta rule: short causal convolutions on q, k and v, unit-norm keys and queries, a decay per head or per key
    channel, gated per-head norm of the read-outs.

    ``forward(h, recur)``: ``recur(pre, z, b)`` advances the sequences' states by the un-convolved rows ``pre (T,
    channels)``, the decay inputs ``z`` and the step-size inputs ``b`` and returns the read-outs, fp32 ``(T, heads, vdim)``."""

    def __init__(self, cfg: DeltaConfig, hidden: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        lin = lambda i, o: nn.Linear(i, o, bias=False)
        kd, vd = cfg.kv_heads * cfg.dim, cfg.heads * cfg.vdim
        self.q_proj, self.k_proj, self.v_proj = lin(hidden, kd), lin(hidden, kd), lin(hidden, vd)
        self.q_conv, self.k_conv = nn.Parameter(torch.zeros(kd, cfg.taps)), nn.Parameter(torch.zeros(kd, cfg.taps))
        self.v_conv = nn.Parameter(torch.zeros(vd, cfg.taps))
        self.beta_proj = lin(hidden, cfg.heads)
        self.A_log, self.dt_bias = nn.Parameter(torch.zeros(cfg.heads)), nn.Parameter(torch.zeros(cfg.decays))
        if cfg.decay_rank:
            self.decay_down, self.decay_up = lin(hidden, cfg.decay_rank), lin(cfg.decay_rank, cfg.decays)
        else:
            self.decay_proj = lin(hidden, cfg.decays)
        if cfg.gate_rank:
            self.gate_down, self.gate_up = lin(hidden, cfg.gate_rank), lin(cfg.gate_rank, vd)
        else:
            self.gate_proj = lin(hidden, vd)
        self.o_norm = nn.Parameter(torch.ones(cfg.vdim))
        self.o_proj = lin(vd, hidden)

    def mix(self, inputs, state, conv, rows, cu_q, past_lens, mask_bits, causal):
        """The recurrence over ``inputs = (pre, z, b)``; states advance when ``causal``."""
        return ops.delta_mix(*inputs, self.conv(), self.A_log, self.dt_bias, self.cfg, state, conv, rows, cu_q, past_lens, mask_bits, causal)

    def conv(self) -> torch.Tensor:
        """Convolution taps of all channels, ``(channels, taps)``, in the order of ``pre``."""
        return torch.cat((self.q_conv, self.k_conv, self.v_conv), 0)

    def forward(self, h, recur):
        c = self.cfg
        lin = ops.linear
        pre = torch.cat([lin(h, p.weight) for p in (self.q_proj, self.k_proj, self.v_proj)], -1)
        b = ops.linear_f32(h, self.beta_proj.weight)
        z = (ops.linear_f32(lin(h, self.decay_down.weight), self.decay_up.weight) if c.decay_rank
             else ops.linear_f32(h, self.decay_proj.weight))
        gate = lin(lin(h, self.gate_down.weight), self.gate_up.weight) if c.gate_rank else lin(h, self.gate_proj.weight)
        y = ops.gated_head_norm(recur(pre, z, b), self.o_norm, gate, c.gate, self.eps)
        return lin(y, self.o_proj.weight)


class Retention(nn.Module):
    """Linear attention with one fixed decay per head: rotated queries and keys, per-head norm of the read-outs without a
    weight, silu gate over all columns.

    ``forward(h, positions, recur)``: ``recur(q, k, v)`` advances the sequences' states by the rotated fp32 rows and returns
    the read-outs, fp32 ``(T, heads, vdim)``."""

    def __init__(self, cfg: RetentionConfig, hidden: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        lin = lambda i, o: nn.Linear(i, o, bias=False)
        self.q_proj, self.k_proj = lin(hidden, cfg.heads * cfg.dim), lin(hidden, cfg.heads * cfg.dim)
        self.v_proj, self.gate_proj = lin(hidden, cfg.heads * cfg.vdim), lin(hidden, cfg.heads * cfg.vdim)
        self.o_proj = lin(cfg.heads * cfg.vdim, hidden)

    def mix(self, inputs, state, conv, rows, cu_q, past_lens, mask_bits, causal):
        """The recurrence over ``inputs = (q, k, v)``; states advance when ``causal``."""
        return ops.retention(*inputs, self.cfg, state, rows, cu_q, past_lens, mask_bits, causal)

    def forward(self, h, positions, recur):
        c, T = self.cfg, h.shape[0]
        q, k = (ops.rotate(ops.linear(h, p.weight).view(T, c.heads, c.dim), positions, c.rot, torch.float32)
                for p in (self.q_proj, self.k_proj))
        o = recur(q.flatten(1), k.flatten(1) * c.dim ** -0.5, ops.linear(h, self.v_proj.weight))
        y = ops.gated_head_norm(o, None, ops.linear(h, self.gate_proj.weight), "silu", self.eps)
        return ops.linear(y, self.o_proj.weight)


class SideBySide(nn.Module):
    """Window attention and a gated delta rule on the same input: half the sum of the two outputs, each RMS-normed over
    the width first.  Returns fp32."""

    def __init__(self, window: WindowAttentionConfig, delta: DeltaConfig, hidden: int, eps: float):
        super().__init__()
        self.left, self.right = WindowAttention(window, hidden, eps), GatedDelta(delta, hidden, eps)
        self.left_norm, self.right_norm = PlainRMSNorm(hidden, eps), PlainRMSNorm(hidden, eps)

    def forward(self, h, positions, attend, recur):
        a = self.left_norm(self.left(h, positions, attend).float())
        return 0.5 * (a + self.right_norm(self.right(h, recur).float()))


class TableMoE(nn.Module):
    """SwiGLU experts named by a table of token ids, equal weights, plus a SwiGLU shared expert.  Returns fp32."""

    def __init__(self, cfg: TableExpertsConfig, hidden: int, vocab: int):
        super().__init__()
        self.cfg = cfg
        self.w_gate, self.w_up = (nn.Parameter(torch.empty(cfg.experts, cfg.ff, hidden)) for _ in range(2))
        self.w_down = nn.Parameter(torch.empty(cfg.experts, hidden, cfg.ff))
        self.register_buffer("table", torch.zeros(vocab, cfg.top, dtype=torch.int32))
        if cfg.shared_ff:
            self.shared_gate, self.shared_up = (nn.Linear(hidden, cfg.shared_ff, bias=False) for _ in range(2))
            self.shared_down = nn.Linear(cfg.shared_ff, hidden, bias=False)

    def forward(self, h, ids):
        y = ops.experts_swiglu(h, self.table[ids], self.w_gate, self.w_up, self.w_down)
        if self.cfg.shared_ff:
            a = torch.cat((ops.linear(h, self.shared_gate.weight), ops.linear(h, self.shared_up.weight)), -1)
            y = y + ops.linear(ops.silu_mul(a), self.shared_down.weight).float()
        return y
