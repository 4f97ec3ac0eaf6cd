"""Op front-end: one function per op, routed to the sm_100a kernel or the reference.

Routing rule: a CUDA bf16 tensor goes to the hand-written kernel in the compiled
extension (and raises if the extension is not loadable — no silent fallback on a
GPU); CPU tensors, and non-bf16 CUDA tensors used by oracle tests, go to the plain
PyTorch implementation in :mod:`jetspec_b200.ops.reference`.  The reference's own seam of this kind is its
``torch.library`` op around the Triton kernel (``jetspec/inference_engine/paged_tree_attn_op.py:29-79``).
"""
from __future__ import annotations

from typing import Optional

import torch

from . import reference as ref
from .reference import (pack_ancestor_bits, unpack_ancestor_bits, rope_cos_sin, apply_rope,
                        moe_route)


def sample(logits, temperature: float = 0.0, generator=None):
    """argmax at temperature 0, else one draw per row from ``softmax(logits / T)``; CUDA tensors use the
    sampling kernel (the generator must then be a CUDA generator or None)."""
    if temperature >= 1e-5 and logits.is_cuda and (generator is None or generator.device.type == "cuda"):
        return _ext().sample_temperature(logits, temperature, generator)
    return ref.sample(logits, temperature, generator)


def _kern(x: torch.Tensor) -> bool:
    return x.is_cuda and x.dtype == torch.bfloat16


def _ext():
    from . import cuda_ext
    return cuda_ext


def rmsnorm(x, weight, eps: float = 1e-6):
    if _kern(x) and x.shape[-1] % 8 == 0:
        return _ext().rmsnorm(x, weight, eps)
    return ref.rmsnorm(x, weight, eps)


def add_rmsnorm(residual, x, weight, eps: float = 1e-6):
    return ref.add_rmsnorm(residual, x, weight, eps)


def linear(x, w, bias: Optional[torch.Tensor] = None):
    if not isinstance(w, torch.Tensor):            # an NVFP4Tensor: 4-bit weights, activations quantised per row
        from ..models.nvfp4 import nvfp4_linear_reference
        if _kern(x) and x.dim() == 2 and w.shape[1] % 256 == 0:
            return _ext().gemm_nvfp4(x.contiguous(), w.swizzled())
        return nvfp4_linear_reference(x, w).to(x.dtype)
    if _kern(x) and bias is None and x.dim() == 2 and w.dtype == torch.bfloat16:
        from . import cuda_ext
        if cuda_ext.gemm_supported(x.shape[0], w.shape[0], x.shape[1]):
            return cuda_ext.gemm(x, w)
    return ref.linear(x, w, bias)


def silu_mul(gate_up):
    if _kern(gate_up) and gate_up.dim() == 2 and gate_up.shape[-1] % 16 == 0:
        return _ext().silu_mul(gate_up)
    return ref.silu_mul(gate_up)


def _kern_any(x: torch.Tensor) -> bool:
    """Ops whose kernels exist in bf16 and in fp32."""
    return x.is_cuda and x.dtype in (torch.bfloat16, torch.float32)


def dynamic_tanh(x, alpha, weight, bias, out_dtype):
    if x.is_cuda and x.dtype == torch.float32 and out_dtype in (torch.bfloat16, torch.float32):
        return _ext().dynamic_tanh(x, alpha, weight, bias, out_dtype)
    return ref.dynamic_tanh(x, alpha, weight, bias, out_dtype)


def gelu_tanh_mul(gate, up):
    if _kern_any(gate):
        return _ext().gelu_tanh_mul(gate, up)
    return ref.gelu_tanh_mul(gate, up)


def relu_squared(x):
    if _kern_any(x):
        return _ext().relu_squared(x)
    return ref.relu_squared(x)


def latent_scatter(c, pool, slots):
    if _kern_any(c):
        return _ext().latent_scatter(c, pool, slots)
    return ref.latent_scatter(c, pool, slots)


def latent_attention(q, w_uk, w_uv, pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale, causal: bool = False, sink=None):
    if _kern_any(q) and pool.shape[1] <= 2048:
        return _ext().latent_attention(q, w_uk, w_uv, pool, slot_map, seq_rows, cu_q, past_lens, mask_bits,
                                       float(scale), bool(causal), sink)
    return ref.latent_attention(q, w_uk, w_uv, pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale, causal, sink)


def sigmoid_moe(x, router_w, correction, w_up, w_down, top, scale):
    if _kern_any(x) and correction.numel() <= 1024 and top <= 32:      # what the routing kernel covers
        wts, idx = _ext().sigmoid_route(ref.linear(x.float(), router_w.float()), correction, top, scale)
        return ref.experts_relu_squared(x, wts, idx.long(), w_up, w_down)
    return ref.sigmoid_moe(x, router_w, correction, w_up, w_down, top, scale)


def rmsnorm_f32(x, weight, eps):
    if x.is_cuda and x.dtype == torch.float32:
        return _ext().rmsnorm_f32(x, weight, eps)
    return ref.rmsnorm_f32(x, weight, eps)


def linear_f32(x, w):
    if _kern(x):
        from . import cuda_ext
        if cuda_ext.gemm_supported(x.shape[0], w.shape[0], x.shape[1]):
            return cuda_ext.gemm(x.contiguous(), w, epi=cuda_ext.EPI_STORE_F32)
    return ref.linear_f32(x, w)


def rotate_norm(x, positions, dims, base, eps):
    if _kern_any(x) and x.shape[-1] <= 512:
        return _ext().rotate_norm(x, positions, dims, base, eps)
    return ref.rotate_norm(x, positions, dims, base, eps)


def window_scatter(k, v, k_pool, v_pool, slots, maps: int = 1):
    return ref.window_scatter(k, v, k_pool, v_pool, slots, maps)


def pool_blocks(k_pool, v_pool, kb_pool, vb_pool, block_map, P, slot_map, seq_rows, cu_q, past_lens):
    if _kern_any(k_pool):
        return _ext().pool_blocks(k_pool, v_pool, kb_pool, vb_pool, block_map, int(P), slot_map, seq_rows, cu_q, past_lens)
    return ref.pool_blocks(k_pool, v_pool, kb_pool, vb_pool, block_map, P, slot_map, seq_rows, cu_q, past_lens)


def window_attention(q, k_pool, v_pool, vdim, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale, window, sink,
                     causal: bool = False, keep_first: int = 0, softcap: float = 0.0, blocks=None, diff=None):
    if _kern_any(q) and max(q.shape[-1], vdim) <= 512:
        return _ext().window_attention(q, k_pool, v_pool, vdim, slot_map, seq_rows, cu_q, past_lens, mask_bits, float(scale),
                                       int(window), sink, bool(causal), keep_first=int(keep_first), softcap=float(softcap),
                                       blocks=blocks, diff=diff)
    return ref.window_attention(q, k_pool, v_pool, vdim, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale, window, sink,
                                causal, keep_first, softcap, blocks, diff)


def query_temperature(x, positions, every, coef):
    return ref.query_temperature(x, positions, every, coef)


def depth_average(history, weights):
    if history[0].is_cuda and history[0].dtype == torch.float32:
        return _ext().depth_average(history, weights)
    return ref.depth_average(history, weights)


def xielu(x, up: float, down: float):
    if _kern_any(x):
        return _ext().xielu(x, up, down)
    return ref.xielu(x, up, down)


def gelu_erf(x):
    if _kern_any(x):
        return _ext().gelu_erf(x)
    return ref.gelu_erf(x)


def rotate(x, positions, rot, out_dtype=None):
    if _kern_any(x) and x.shape[-1] <= 1024 and (out_dtype or x.dtype) in (torch.bfloat16, torch.float32):
        return _ext().rotate(x, positions, rot, out_dtype or x.dtype)
    return ref.rotate(x, positions, rot, out_dtype)


def head_gate(y, logits):
    if _kern_any(y):
        return _ext().head_gate(y, logits)
    return ref.head_gate(y, logits)


def retention(q, k, v, cfg, state, rows, cu_q, past_lens, mask_bits, causal: bool = True):
    if _kern_any(q) and cfg.dim <= 256 and (causal or mask_bits.shape[1] <= 8):
        return _ext().retention(q, k, v, cfg, state, rows, cu_q, past_lens, mask_bits, bool(causal))
    return ref.retention(q, k, v, cfg, state, rows, cu_q, past_lens, mask_bits, causal)


def delta_mix(pre, z, b, taps, A_log, dt_bias, cfg, state, conv, rows, cu_q, past_lens, mask_bits, causal: bool = True):
    if _kern_any(pre) and cfg.dim <= 256 and cfg.taps <= 17:
        return _ext().delta_mix(pre, z, b, taps, A_log, dt_bias, cfg, state, conv, rows, cu_q, past_lens, mask_bits,
                                bool(causal))
    return ref.delta_mix(pre, z, b, taps, A_log, dt_bias, cfg, state, conv, rows, cu_q, past_lens, mask_bits, causal)


def gated_head_norm(o, weight, gate, kind, eps):
    if _kern_any(gate):
        return _ext().gated_head_norm(o, weight, gate, kind, eps)
    return ref.gated_head_norm(o, weight, gate, kind, eps)


def experts_swiglu(x, idx, w_gate, w_up, w_down):
    return ref.experts_swiglu(x, idx, w_gate, w_up, w_down)


def qkv_postprocess(qkv, q_norm_w, k_norm_w, positions, num_q_heads, num_kv_heads, head_dim, theta, eps):
    if _kern(qkv) and head_dim == 128:
        ext = _ext()
        T = qkv.shape[0]
        q = torch.empty(T, num_q_heads, head_dim, dtype=qkv.dtype, device=qkv.device)
        k = torch.empty(num_kv_heads, T, head_dim, dtype=qkv.dtype, device=qkv.device)
        v = torch.empty_like(k)
        rows = torch.arange(T, dtype=torch.int32, device=qkv.device)
        ext.qkv_post(qkv, q_norm_w, k_norm_w, positions.to(torch.int32), rows,
                     ext.inv_freq(head_dim, theta, qkv.device), q, k, v, num_q_heads, num_kv_heads, float(eps))
        return q, k.transpose(0, 1), v.transpose(0, 1)
    return ref.qkv_postprocess(qkv, q_norm_w, k_norm_w, positions, num_q_heads, num_kv_heads,
                               head_dim, theta, eps)


def kv_scatter(k, v, k_pool, v_pool, slots):
    return ref.kv_scatter(k, v, k_pool, v_pool, slots)


def paged_tree_attention(q, k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens, mask_bits, scale,
                         causal: bool = False, max_q: Optional[int] = None):
    if _kern(q) and q.shape[-1] == 128:
        return _ext().paged_tree_attention(q.contiguous(), k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens,
                                           mask_bits, float(scale), bool(causal),
                                           int(max_q if max_q is not None else q.shape[0]))
    return ref.paged_tree_attention(q, k_pool, v_pool, slot_map, seq_rows, cu_q, past_lens,
                                    mask_bits, scale, causal)


def lm_head_argmax(h, w):
    if _kern(h):
        from . import cuda_ext
        return cuda_ext.lm_head_argmax(h, w)
    return ref.lm_head_argmax(h, w)


def lm_head_topk_logprobs(h, w, k: int):
    if _kern(h):
        from . import cuda_ext
        return cuda_ext.lm_head_topk_logprobs(h, w, k)
    return ref.lm_head_topk_logprobs(h, w, k)


def moe_forward(x, gate_w, w_gate_up, w_down, top_k, renorm, router_logits=None):
    if _kern(x):
        from . import cuda_ext
        return cuda_ext.moe_forward(x, gate_w, w_gate_up, w_down, top_k, renorm, router_logits)
    return ref.moe_forward(x, gate_w, w_gate_up, w_down, top_k, renorm, router_logits)


__all__ = [
    "rmsnorm", "add_rmsnorm", "linear", "silu_mul", "qkv_postprocess", "kv_scatter",
    "paged_tree_attention", "lm_head_argmax", "lm_head_topk_logprobs", "moe_forward",
    "dynamic_tanh", "gelu_tanh_mul", "relu_squared", "latent_scatter", "latent_attention", "sigmoid_moe",
    "rmsnorm_f32", "linear_f32", "rotate_norm", "window_scatter", "window_attention", "delta_mix", "gated_head_norm",
    "experts_swiglu", "pool_blocks", "query_temperature", "depth_average", "xielu", "gelu_erf", "rotate", "head_gate", "retention",
    "pack_ancestor_bits", "unpack_ancestor_bits", "rope_cos_sin", "apply_rope", "moe_route", "sample",
]
