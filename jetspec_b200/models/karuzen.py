"""Karuzen decoder: parallel blocks, Dynamic Tanh norms, latent attention, looped layers, tied embeddings.

A block normalises the fp32 residual stream once, hands the result to its mixer and its feed-forward side by side and
adds what both return.  A range of blocks can be traversed repeatedly with shared weights; each traversal writes cache
layers of its own, and every later one starts by adding the token embeddings to the stream.  ``forward`` has the contract of
:meth:`jetspec_b200.models.qwen3.Qwen3ForCausalLM.forward`, so the engines drive both families alike; layer numbers
(taps, cache layers) count layer RUNS.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn as nn

from .. import ops
from .config import KaruzenConfig
from .layers import DynamicTanh, GeluMLP, LatentAttention, SigmoidMoE
from .qwen3 import _fill_normal_
from .registry import register_family


class KaruzenLayer(nn.Module):
    def __init__(self, cfg: KaruzenConfig, i: int):
        super().__init__()
        l = cfg.layers[i]
        self.norm = DynamicTanh(cfg.hidden_size)
        self.mixer = LatentAttention(l.mixer, cfg.hidden_size, cfg.norm_eps)
        self.mlp = (GeluMLP(cfg.hidden_size, l.dense_ff) if l.dense_ff
                    else SigmoidMoE(l.moe, cfg.hidden_size) if l.moe is not None else None)


class KaruzenModel(nn.Module):
    def __init__(self, cfg: KaruzenConfig):
        super().__init__()
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size)
        self.layers = nn.ModuleList(KaruzenLayer(cfg, i) for i in range(len(cfg.layers)))
        self.norm = DynamicTanh(cfg.hidden_size)


# checkpoint name below ``l<i>.`` -> parameter below ``model.layers.<i>.``
_LAYER_NAMES = {
    "norm1": "norm.weight", "norm1.b": "norm.bias", "norm1.alpha": "norm.alpha",
    "mix.dq": "mixer.q_down.weight", "mix.dq.norm": "mixer.q_norm", "mix.uq": "mixer.q_up.weight",
    "mix.dkv": "mixer.kv_down.weight", "mix.dkv.norm": "mixer.kv_norm", "mix.uk": "mixer.k_up.weight",
    "mix.uv": "mixer.v_up.weight", "mix.o": "mixer.o_proj.weight",
    "mlp.gate": "mlp.gate_proj.weight", "mlp.up": "mlp.up_proj.weight", "mlp.down": "mlp.down_proj.weight",
    "mlp.router": "mlp.router.weight", "mlp.correction": "mlp.correction",
    "mlp.shared.up": "mlp.shared_up.weight", "mlp.shared.down": "mlp.shared_down.weight",
    "mlp.shared.sg": "mlp.shared_gate.weight",
}
_TOP_NAMES = {"embed": "model.embed_tokens.weight", "final.norm": "model.norm.weight", "final.norm.b": "model.norm.bias",
              "final.norm.alpha": "model.norm.alpha"}


def checkpoint_to_parameter(key: str):
    """``(parameter name, index or None)`` of a checkpoint tensor; experts land in the stacked parameters."""
    if key in _TOP_NAMES:
        return _TOP_NAMES[key], None
    head, _, rest = key.partition(".")
    if not (head[:1] == "l" and head[1:].isdigit()):
        return key, None
    base = f"model.layers.{head[1:]}."
    if rest in _LAYER_NAMES:
        return base + _LAYER_NAMES[rest], None
    parts = rest.split(".")
    if len(parts) == 3 and parts[0] == "mlp" and parts[1][:1] == "e" and parts[1][1:].isdigit() and parts[2] in ("up", "down"):
        return base + f"mlp.w_{parts[2]}", (int(parts[1][1:]),)
    return key, None


class KaruzenForCausalLM(nn.Module):
    """Decoder-only LM.  ``forward`` is token-major and cache-agnostic."""

    def __init__(self, cfg: KaruzenConfig):
        super().__init__()
        self.config = cfg
        self.model = KaruzenModel(cfg)
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
    def random_init(cls, cfg: KaruzenConfig, seed: int = 0, dtype=torch.float32, device="cpu", std: float = 0.02,
                    init: str = "normal") -> "KaruzenForCausalLM":
        """Synthetic weights.  ``"normal"``: matrices N(0, std), norm scales 1, ``alpha`` 0.5.  ``"stable"``: embedding
        N(0, 1) and output projections scaled down by ``sqrt(2 runs)``, so that the residual stream stays close to
        the token's own embedding and the greedy choice has a wide margin (see ``Qwen3ForCausalLM.random_init``)."""
        m = cls._empty(cfg, dtype, device)
        g = torch.Generator(device="cpu").manual_seed(seed)
        out_scale = 1.0 / (2.0 * cfg.num_hidden_layers) ** 0.5
        with torch.no_grad():
            for name, p in m.named_parameters():
                leaf = name.rsplit(".", 1)[-1]
                if leaf == "alpha":
                    p.fill_(0.5)
                elif name.endswith("norm.weight") or leaf in ("q_norm", "kv_norm"):
                    p.fill_(1.0)
                elif leaf in ("bias", "correction"):
                    p.zero_()
                elif init == "stable" and name.endswith("embed_tokens.weight"):
                    _fill_normal_(p, 1.0, g)
                elif init == "stable" and ("o_proj" in name or "down_proj" in name or "shared_down" in name or leaf == "w_down"):
                    _fill_normal_(p, std * out_scale, g)
                else:
                    _fill_normal_(p, std, g)
        return m.eval()

    @classmethod
    def from_pretrained(cls, path: str, dtype=torch.bfloat16, device="cpu") -> "KaruzenForCausalLM":
        from .loader import load_state_into
        m = cls._empty(KaruzenConfig.from_pretrained(path), dtype, device)
        load_state_into(m, path, remap=checkpoint_to_parameter)
        return m.eval()

    def save_pretrained(self, path: str) -> None:
        from .loader import save_state
        self.config.save_pretrained(path)
        params = dict(self.named_parameters())
        sd = {k: params[v] for k, v in _TOP_NAMES.items()}
        for i, layer in enumerate(self.config.layers):
            base = f"model.layers.{i}."
            sd.update({f"l{i}.{k}": params[base + v] for k, v in _LAYER_NAMES.items() if base + v in params})
            if layer.moe is not None:
                for e in range(layer.moe.experts):
                    sd[f"l{i}.mlp.e{e}.up"] = params[base + "mlp.w_up"][e]
                    sd[f"l{i}.mlp.e{e}.down"] = params[base + "mlp.w_down"][e]
        save_state(sd, path)

    # -- forward ----------------------------------------------------------------
    @torch.inference_mode()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, attn, tap_layers: Optional[Sequence[int]] = None,
                logits_rows=None, router_logits_fn=None, return_hidden: bool = False):
        """Run the decoder on ``input_ids (T,)``.

        ``attn.latent(run, mixer, q, c)`` stores the latent rows of layer run ``run`` and attends over them; the design
        uses no positions beyond the cache's order, so ``positions`` only keeps the common signature.  ``tap_layers``
        are layer runs; the last one is tapped after the final norm.  Returns ``(logits, taps or None)``."""
        emb = self.model.embed_tokens.weight[input_ids].float()
        x = emb
        dtype = self.model.embed_tokens.weight.dtype
        runs = self.config.layer_runs()
        tap_ids = list(tap_layers) if tap_layers is not None else None
        tapped = {}
        for run, (i, again) in enumerate(runs):
            layer = self.model.layers[i]
            if again:
                x = x + emb
            h = layer.norm(x, dtype)
            y = layer.mixer(h, lambda q, c: attn.latent(run, layer.mixer, q, c)).float()
            if layer.mlp is not None:
                y = y + layer.mlp(h).float()
            x = x + y
            if tap_ids is not None and run in tap_ids:
                tapped[run] = x.to(dtype)
        xn = self.model.norm(x, dtype)
        if tap_ids is not None and len(runs) - 1 in tap_ids:
            tapped[len(runs) - 1] = xn
        tap_cat = torch.cat([tapped[t] for t in tap_ids], dim=-1) if tap_ids else None
        rows = xn if logits_rows is None else xn[logits_rows]
        logits = ops.linear(rows, self.lm_head.weight)
        if return_hidden:
            return logits, tap_cat, xn
        return logits, tap_cat


register_family("karuzen", KaruzenConfig, KaruzenForCausalLM, aliases=("Karuzen", "KaruzenForCausalLM"))
