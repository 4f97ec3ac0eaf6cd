"""Sogidra decoder: differential attention over the whole past and window attention with pooled blocks, in any order.

Every sublayer is normed on both sides, and what a layer passes on is a weighted sum of the embedding output and all layers'
results so far.  A layer may attend with its own queries over an earlier layer's keys and values.  Sequence memory is a paged
K/V cache, with one row more per whole block where a layer pools blocks (see :mod:`jetspec_b200.runtime.kv_pool`).  The residual
stream is fp32.  ``forward`` takes and returns what :meth:`jetspec_b200.models.qwen3.Qwen3ForCausalLM.forward` does, so the
engines drive every family alike.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn as nn

from .. import ops
from .config import SogidraConfig
from .layers import OffsetRMSNorm, WindowAttention, XieluMLP
from .qwen3 import _fill_normal_
from .registry import register_family


class SogidraLayer(nn.Module):
    def __init__(self, cfg: SogidraConfig, i: int):
        super().__init__()
        l, W, eps = cfg.layers[i], cfg.hidden_size, cfg.norm_eps
        self.norm1, self.norm1b = OffsetRMSNorm(W, eps), OffsetRMSNorm(W, eps)
        self.mixer = WindowAttention(l.mixer, W, eps)
        self.mlp = XieluMLP(W, l.ff) if l.ff else None
        if l.ff:
            self.norm2, self.norm2b = OffsetRMSNorm(W, eps), OffsetRMSNorm(W, eps)
        self.dwa = nn.Parameter(torch.zeros(i + 2))


class SogidraModel(nn.Module):
    def __init__(self, cfg: SogidraConfig):
        super().__init__()
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size)
        self.pos_embed = nn.Embedding(cfg.max_positions, cfg.hidden_size)
        self.layers = nn.ModuleList(SogidraLayer(cfg, i) for i in range(len(cfg.layers)))
        self.norm = OffsetRMSNorm(cfg.hidden_size, cfg.norm_eps)


# checkpoint name below a layer -> parameter below it
_LAYER_NAMES = {**{n: f"{n}.weight" for n in ("norm1", "norm1b", "norm2", "norm2b")}, "dwa": "dwa",
                **{f"mix.{n}": f"mixer.{n}_proj.weight" for n in "qkvo"}, **{f"mix.{n}.b": f"mixer.{n}_proj.bias" for n in "qkv"},
                **{f"mix.{n}": f"mixer.{n}" for n in ("lq1", "lk1", "lq2", "lk2")},
                "mlp.up": "mlp.up_proj.weight", "mlp.down": "mlp.down_proj.weight", "mlp.act": "mlp.act"}
_TOP_NAMES = {"embed": "model.embed_tokens.weight", "pos": "model.pos_embed.weight", "final.norm": "model.norm.weight"}


def checkpoint_to_parameter(key: str):
    """``(parameter name, None)`` of a checkpoint name."""
    if key in _TOP_NAMES:
        return _TOP_NAMES[key], None
    head, _, rest = key.partition(".")
    if head[:1] == "l" and head[1:].isdigit() and rest in _LAYER_NAMES:
        return f"model.layers.{int(head[1:])}.{_LAYER_NAMES[rest]}", None
    return key, None


class SogidraForCausalLM(nn.Module):
    """Decoder-only LM.  ``forward`` is token-major and cache-agnostic."""

    def __init__(self, cfg: SogidraConfig):
        super().__init__()
        self.config = cfg
        self.model = SogidraModel(cfg)
        self.lm_head = nn.Linear(cfg.hidden_size, cfg.vocab_size, bias=False)
        self.lm_head.weight = self.model.embed_tokens.weight

    # -- construction ---------------------------------------------------------
    @classmethod
    def _empty(cls, cfg, dtype, device):
        with torch.device("meta"):
            m = cls(cfg)
        m = m.to_empty(device=device).to(dtype)
        m.lm_head.weight = m.model.embed_tokens.weight
        return m

    @classmethod
    def random_init(cls, cfg: SogidraConfig, seed: int = 0, dtype=torch.float32, device="cpu", std: float = 0.02,
                    init: str = "normal") -> "SogidraForCausalLM":
        """Synthetic weights.  ``"normal"``: matrices N(0, std), norms 1, biases 0, a layer passes its own result on.
        ``"stable"``: embedding N(0, 1) and small norms behind the sublayers, so that the stream stays close to the token's own
        embedding and the greedy choice has a wide margin."""
        m = cls._empty(cfg, dtype, device)
        g = torch.Generator(device="cpu").manual_seed(seed)
        with torch.no_grad():
            for name, p in m.named_parameters():
                if name.endswith(("norm1b.weight", "norm2b.weight")):
                    p.fill_(-0.96875 if init == "stable" else 0.0)
                elif "norm" in name or name.endswith(("bias", ".act", "lq1", "lk1", "lq2", "lk2")):
                    p.zero_()
                elif name.endswith("dwa"):
                    p.zero_()
                    p[-1] = 1.0
                elif init == "stable" and name.endswith("embed_tokens.weight"):
                    _fill_normal_(p, 1.0, g)
                else:
                    _fill_normal_(p, std, g)
        return m.eval()

    @classmethod
    def from_pretrained(cls, path: str, dtype=torch.bfloat16, device="cpu") -> "SogidraForCausalLM":
        from .loader import load_state_into
        m = cls._empty(SogidraConfig.from_pretrained(path), dtype, device)
        load_state_into(m, path, remap=checkpoint_to_parameter)
        return m.eval()

    def save_pretrained(self, path: str) -> None:
        from .loader import save_state
        self.config.save_pretrained(path)
        params = self.state_dict()
        sd = {k: params[v] for k, v in _TOP_NAMES.items()}
        for i in range(len(self.config.layers)):
            base = f"model.layers.{i}."
            sd.update({f"l{i}.{k}": params[base + v] for k, v in _LAYER_NAMES.items() if base + v in params})
        save_state(sd, path)

    # -- forward ----------------------------------------------------------------
    @torch.inference_mode()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, attn, tap_layers: Optional[Sequence[int]] = None,
                logits_rows=None, router_logits_fn=None, return_hidden: bool = False):
        """Run the decoder on ``input_ids (T,)``.

        ``attn.window(layer, mixer, q, k, v)`` stores K/V rows (unless they are ``None``) and attends.  Layers are tapped behind
        their depth average, the last one after the final norm.  Positions past the table (nodes of a token tree no request can
        keep) take its last row.  Returns ``(logits, taps or None)``."""
        dtype, table = self.model.embed_tokens.weight.dtype, self.model.pos_embed.weight
        x = self.model.embed_tokens.weight[input_ids].float() + table[positions.clamp(max=table.shape[0] - 1)].float()
        history = [x]
        tap_ids = list(tap_layers) if tap_layers is not None else None
        tapped, last = {}, len(self.model.layers) - 1
        for i, layer in enumerate(self.model.layers):
            mix = layer.mixer
            y = mix(layer.norm1(x).to(dtype), positions, lambda q, k, v: attn.window(i, mix, q, k, v))
            x = x + layer.norm1b(y.float())
            if layer.mlp is not None:
                x = x + layer.norm2b(layer.mlp(layer.norm2(x).to(dtype)).float())
            history.append(x)
            x = ops.depth_average(history, layer.dwa)
            if tap_ids is not None and i in tap_ids:
                tapped[i] = x.to(dtype)
        xn = self.model.norm(x).to(dtype)
        if tap_ids is not None and last in tap_ids:
            tapped[last] = xn
        tap_cat = torch.cat([tapped[t] for t in tap_ids], dim=-1) if tap_ids else None
        rows = xn if logits_rows is None else xn[logits_rows]
        logits = ops.linear(rows, self.lm_head.weight)
        if return_hidden:
            return logits, tap_cat, xn
        return logits, tap_cat


register_family("sogidra", SogidraConfig, SogidraForCausalLM, aliases=("Sogidra", "SogidraForCausalLM"))
