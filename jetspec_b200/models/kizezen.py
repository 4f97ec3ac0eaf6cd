"""Kizezen decoder: pre-norm blocks whose mixers are window attention, latent attention or retention, in any order.

A layer's sequence memory is a paged K/V cache (window attention), paged latent rows (latent attention) or a recurrent state
(retention), see :mod:`jetspec_b200.runtime.kv_pool` and :mod:`jetspec_b200.runtime.state_pool`.  The residual stream is fp32.
``forward`` has the contract of :meth:`jetspec_b200.models.qwen3.Qwen3ForCausalLM.forward`, so the engines drive every family
alike.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn as nn

from .. import ops
from .config import KizezenConfig, LatentAttentionConfig, RetentionConfig, WindowAttentionConfig
from .layers import GeluErfMLP, LatentAttention, PlainRMSNorm, Retention, WindowAttention
from .qwen3 import _fill_normal_
from .registry import register_family

_MIXERS = {WindowAttentionConfig: WindowAttention, LatentAttentionConfig: LatentAttention, RetentionConfig: Retention}


class KizezenLayer(nn.Module):
    def __init__(self, cfg: KizezenConfig, i: int):
        super().__init__()
        l, W, eps = cfg.layers[i], cfg.hidden_size, cfg.norm_eps
        self.norm1 = PlainRMSNorm(W, eps)
        self.mixer = _MIXERS[type(l.mixer)](l.mixer, W, eps)
        self.mlp = GeluErfMLP(W, l.ff) if l.ff else None
        if l.ff:
            self.norm2 = PlainRMSNorm(W, eps)


class KizezenModel(nn.Module):
    def __init__(self, cfg: KizezenConfig):
        super().__init__()
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size)
        self.layers = nn.ModuleList(KizezenLayer(cfg, i) for i in range(len(cfg.layers)))
        self.norm = PlainRMSNorm(cfg.hidden_size, cfg.norm_eps)


# checkpoint name below a layer -> parameter below it
_COMMON = {"norm1": "norm1.weight", "norm2": "norm2.weight", "mlp.up": "mlp.up_proj.weight", "mlp.down": "mlp.down_proj.weight",
           "mix.q": "mixer.q_proj.weight", "mix.g": "mixer.gate_proj.weight", "mix.o": "mixer.o_proj.weight"}
_KV = {"mix.k": "mixer.k_proj.weight", "mix.v": "mixer.v_proj.weight"}
_LAYER_NAMES = {
    "attention": {**_COMMON, **_KV, **{f"mix.{n}.b": f"mixer.{n}_proj.bias" for n in "qkv"},
                  "mix.q.norm": "mixer.q_norm", "mix.k.norm": "mixer.k_norm", "mix.sink": "mixer.sink_logits"},
    "latent_attention": {**_COMMON, "mix.dkv": "mixer.kv_down.weight", "mix.dkv.norm": "mixer.kv_norm", "mix.uk": "mixer.k_up.weight",
                         "mix.uv": "mixer.v_up.weight", "mix.sink": "mixer.sink"},
    "retention": {**_COMMON, **_KV},
}
_TOP_NAMES = {"embed": "model.embed_tokens.weight", "final.norm": "model.norm.weight", "head": "lm_head.weight"}


def checkpoint_to_parameter(cfg: KizezenConfig):
    """``remap(checkpoint name) -> (parameter name, None)`` for a model of ``cfg``."""
    def remap(key: str):
        if key in _TOP_NAMES:
            return _TOP_NAMES[key], None
        head, _, rest = key.partition(".")
        if head[:1] == "l" and head[1:].isdigit() and int(head[1:]) < len(cfg.layers):
            name = _LAYER_NAMES[cfg.layers[int(head[1:])].mixer_type].get(rest)
            if name is not None:
                return f"model.layers.{int(head[1:])}.{name}", None
        return key, None
    return remap


class KizezenForCausalLM(nn.Module):
    """Decoder-only LM.  ``forward`` is token-major and cache-agnostic."""

    def __init__(self, cfg: KizezenConfig):
        super().__init__()
        self.config = cfg
        self.model = KizezenModel(cfg)
        self.lm_head = nn.Linear(cfg.hidden_size, cfg.vocab_size, bias=False)

    # -- construction ---------------------------------------------------------
    @classmethod
    def _empty(cls, cfg, dtype, device):
        with torch.device("meta"):
            m = cls(cfg)
        return m.to_empty(device=device).to(dtype)

    @classmethod
    def random_init(cls, cfg: KizezenConfig, seed: int = 0, dtype=torch.float32, device="cpu", std: float = 0.02,
                    init: str = "normal") -> "KizezenForCausalLM":
        """Synthetic weights.  ``"normal"``: matrices N(0, std), norms 1, biases and sinks 0.  ``"stable"``: embedding and
        head N(0, 1) and equal, output projections scaled down, so that the stream stays close to the token's own embedding
        and the greedy choice has a wide margin."""
        m = cls._empty(cfg, dtype, device)
        g = torch.Generator(device="cpu").manual_seed(seed)
        with torch.no_grad():
            for name, p in m.named_parameters():
                if "norm" in name:
                    p.fill_(1.0)
                elif name.endswith(("bias", "sink", "sink_logits")):
                    p.zero_()
                elif init == "stable" and name.endswith(("embed_tokens.weight", "lm_head.weight")):
                    _fill_normal_(p, 1.0, torch.Generator(device="cpu").manual_seed(seed))
                elif init == "stable" and name.endswith(("o_proj.weight", "down_proj.weight")):
                    _fill_normal_(p, std / (2.0 * cfg.num_hidden_layers) ** 0.5, g)
                else:
                    _fill_normal_(p, std, g)
        return m.eval()

    @classmethod
    def from_pretrained(cls, path: str, dtype=torch.bfloat16, device="cpu") -> "KizezenForCausalLM":
        from .loader import load_state_into
        cfg = KizezenConfig.from_pretrained(path)
        m = cls._empty(cfg, dtype, device)
        load_state_into(m, path, remap=checkpoint_to_parameter(cfg), optional=())       # the head is a tensor of its own
        return m.eval()

    def save_pretrained(self, path: str) -> None:
        from .loader import save_state
        self.config.save_pretrained(path)
        params = self.state_dict()
        sd = {k: params[v] for k, v in _TOP_NAMES.items()}
        for i, layer in enumerate(self.config.layers):
            base = f"model.layers.{i}."
            sd.update({f"l{i}.{k}": params[base + v] for k, v in _LAYER_NAMES[layer.mixer_type].items() if base + v in params})
        save_state(sd, path)

    # -- forward ----------------------------------------------------------------
    @torch.inference_mode()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, attn, tap_layers: Optional[Sequence[int]] = None,
                logits_rows=None, router_logits_fn=None, return_hidden: bool = False):
        """Run the decoder on ``input_ids (T,)``.

        ``attn.window(layer, mixer, q, k, v)`` and ``attn.latent(layer, mixer, q, c)`` store cache rows and attend,
        ``attn.recur(layer, mixer, q, k, v)`` advances a retention's states.  The last tapped layer is tapped after the final
        norm.  Returns ``(logits, taps or None)``."""
        cfg, dtype = self.config, self.model.embed_tokens.weight.dtype
        x = self.model.embed_tokens.weight[input_ids].float() * cfg.embed_scale
        tap_ids = list(tap_layers) if tap_layers is not None else None
        tapped, last = {}, len(self.model.layers) - 1
        for i, layer in enumerate(self.model.layers):
            mix, h = layer.mixer, layer.norm1(x).to(dtype)
            if isinstance(mix, WindowAttention):
                y = mix(h, positions, lambda q, k, v: attn.window(i, mix, q, k, v))
            elif isinstance(mix, LatentAttention):
                y = mix(h, lambda q, c: attn.latent(i, mix, q, c), positions)
            else:
                y = mix(h, positions, lambda q, k, v: attn.recur(i, mix, q, k, v))
            x = x + y.float()
            if layer.mlp is not None:
                x = x + layer.mlp(layer.norm2(x).to(dtype)).float()
            if tap_ids is not None and i in tap_ids:
                tapped[i] = x.to(dtype)
        xn = self.model.norm(x).to(dtype)
        if tap_ids is not None and last in tap_ids:
            tapped[last] = xn
        tap_cat = torch.cat([tapped[t] for t in tap_ids], dim=-1) if tap_ids else None
        rows = xn if logits_rows is None else xn[logits_rows]
        logits = ops.linear(rows, self.lm_head.weight) * cfg.logit_scale
        if return_hidden:
            return logits, tap_cat, xn
        return logits, tap_cat


register_family("kizezen", KizezenConfig, KizezenForCausalLM, aliases=("Kizezen", "KizezenForCausalLM"))
