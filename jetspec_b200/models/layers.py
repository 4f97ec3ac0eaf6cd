"""Building blocks that are not Qwen3's: Dynamic Tanh, latent attention, tanh-GELU MLP, sigmoid-routed experts.

Each takes its sizes and constants as arguments, so a design can combine them freely; the Qwen3 twins (RMSNorm, grouped
query attention, SwiGLU MLP, softmax-routed experts) are in :mod:`jetspec_b200.models.qwen3`.  ``forward`` is the
unfused form on :mod:`jetspec_b200.ops`, in any dtype and on any device; the fused kernel form of a whole decoder made
of these blocks is :mod:`jetspec_b200.engine.latent_stack`.
"""
from __future__ import annotations

import torch
import torch.nn as nn

from .. import ops
from .config import LatentAttentionConfig, RoutedExpertsConfig


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
    """Attention whose queries and keys/values pass through RMS-normed latents; only the K/V latent is cached.

    ``forward(h, attend)``: ``attend(q, c)`` stores the new latent rows ``c (T, kv_rank)`` and returns the attention of
    ``q (T, heads, dim)`` over the cached latents, ``(T, heads * vdim)``."""

    def __init__(self, cfg: LatentAttentionConfig, hidden: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        lin = lambda i, o: nn.Linear(i, o, bias=False)
        self.q_down, self.q_up = lin(hidden, cfg.q_rank), lin(cfg.q_rank, cfg.heads * cfg.dim)
        self.kv_down = lin(hidden, cfg.kv_rank)
        self.k_up, self.v_up = lin(cfg.kv_rank, cfg.heads * cfg.dim), lin(cfg.kv_rank, cfg.heads * cfg.vdim)
        self.o_proj = lin(cfg.heads * cfg.vdim, hidden)
        self.q_norm, self.kv_norm = nn.Parameter(torch.ones(cfg.q_rank)), nn.Parameter(torch.ones(cfg.kv_rank))

    def forward(self, h, attend):
        m = self.cfg
        cq = ops.rmsnorm(ops.linear(h, self.q_down.weight), self.q_norm, self.eps)
        c = ops.rmsnorm(ops.linear(h, self.kv_down.weight), self.kv_norm, self.eps)
        q = ops.linear(cq, self.q_up.weight).view(h.shape[0], m.heads, m.dim)
        return ops.linear(attend(q, c), self.o_proj.weight)


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
