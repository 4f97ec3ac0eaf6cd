"""Zasipel decoder: window attention beside a gated delta rule, channel-decay delta layers, experts chosen by token id.

The sublayers read the fp32 residual stream itself; each one's output is RMS-normed before it is added.  A layer's
sequence memory is a paged K/V cache (window attention) and a recurrent state (delta rules), see
:mod:`jetspec_b200.runtime.kv_pool` and :mod:`jetspec_b200.runtime.state_pool`.  ``forward`` has the contract of
:meth:`jetspec_b200.models.qwen3.Qwen3ForCausalLM.forward`, so the engines drive every family alike.
"""
from __future__ import annotations

from typing import Optional, Sequence

import torch
import torch.nn as nn

from .. import ops
from .config import ZasipelConfig
from .layers import GatedDelta, PlainRMSNorm, SideBySide, TableMoE
from .qwen3 import _fill_normal_
from .registry import register_family


class ZasipelLayer(nn.Module):
    def __init__(self, cfg: ZasipelConfig, i: int):
        super().__init__()
        l, W, eps = cfg.layers[i], cfg.hidden_size, cfg.norm_eps
        self.mixer = SideBySide(l.window, l.delta, W, eps) if l.window is not None else GatedDelta(l.delta, W, eps)
        self.norm1 = PlainRMSNorm(W, eps)
        self.mlp = TableMoE(l.moe, W, cfg.vocab_size) if l.moe is not None else None
        if l.moe is not None:
            self.norm2 = PlainRMSNorm(W, eps)

    @property
    def delta(self) -> GatedDelta:
        return self.mixer.right if isinstance(self.mixer, SideBySide) else self.mixer


class ZasipelModel(nn.Module):
    def __init__(self, cfg: ZasipelConfig):
        super().__init__()
        self.embed_tokens = nn.Embedding(cfg.vocab_size, cfg.hidden_size)
        self.layers = nn.ModuleList(ZasipelLayer(cfg, i) for i in range(len(cfg.layers)))
        self.norm = PlainRMSNorm(cfg.hidden_size, cfg.norm_eps)


# checkpoint name below a mixer -> parameter below it
_WINDOW_NAMES = {f"{a}{b}": f"{a}_proj.{c}" for a in "qkvo" for b, c in (("", "weight"), (".b", "bias"))}
_DELTA_NAMES = {**{a: f"{a}_proj.weight" for a in "qkvo"}, **{f"{a}.conv": f"{a}_conv" for a in "qkv"},
                "b": "beta_proj.weight", "a": "decay_proj.weight", "a1": "decay_down.weight", "a2": "decay_up.weight",
                "g": "gate_proj.weight", "g1": "gate_down.weight", "g2": "gate_up.weight",
                "A_log": "A_log", "dt_bias": "dt_bias", "norm": "o_norm"}
_LAYER_NAMES = {
    "norm1": "norm1.weight", "norm2": "norm2.weight",
    "mix.left.out": "mixer.left_norm.weight", "mix.right.out": "mixer.right_norm.weight",
    **{f"mix.left.{k}": f"mixer.left.{v}" for k, v in _WINDOW_NAMES.items()},
    **{f"mix.right.{k}": f"mixer.right.{v}" for k, v in _DELTA_NAMES.items()},
    **{f"mix.{k}": f"mixer.{v}" for k, v in _DELTA_NAMES.items()},
    "mlp.table": "mlp.table", "mlp.shared.gate": "mlp.shared_gate.weight", "mlp.shared.up": "mlp.shared_up.weight",
    "mlp.shared.down": "mlp.shared_down.weight",
}
_TOP_NAMES = {"embed": "model.embed_tokens.weight", "final.norm": "model.norm.weight", "head": "lm_head.weight"}
_EXPERT_PARTS = ("gate", "up", "down")


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
    if len(parts) == 3 and parts[0] == "mlp" and parts[1][:1] == "e" and parts[1][1:].isdigit() and parts[2] in _EXPERT_PARTS:
        return base + f"mlp.w_{parts[2]}", (int(parts[1][1:]),)
    return key, None


class ZasipelForCausalLM(nn.Module):
    """Decoder-only LM.  ``forward`` is token-major and cache-agnostic."""

    def __init__(self, cfg: ZasipelConfig):
        super().__init__()
        self.config = cfg
        self.model = ZasipelModel(cfg)
        self.lm_head = nn.Linear(cfg.hidden_size, cfg.vocab_size, bias=False)

    # -- construction ---------------------------------------------------------
    @classmethod
    def _empty(cls, cfg, dtype, device):
        with torch.device("meta"):
            m = cls(cfg)
        return m.to_empty(device=device).to(dtype)

    @classmethod
    def random_init(cls, cfg: ZasipelConfig, seed: int = 0, dtype=torch.float32, device="cpu", std: float = 0.02,
                    init: str = "normal") -> "ZasipelForCausalLM":
        """Synthetic weights.  ``"normal"``: matrices N(0, std), norms 1, taps on the current token, decays spread over
        short and long memories.  ``"stable"``: embedding and head N(0, 1) and equal, output norms small, so that the
        stream stays close to the token's own embedding and the greedy choice has a wide margin."""
        m = cls._empty(cfg, dtype, device)
        g = torch.Generator(device="cpu").manual_seed(seed)
        with torch.no_grad():
            for name, p in m.named_parameters():
                leaf = name.rsplit(".", 1)[-1]
                if leaf == "A_log":
                    p.copy_(torch.linspace(-4.0, 0.0, p.numel()))
                elif leaf == "dt_bias":
                    p.fill_(-2.0)
                elif leaf.endswith("_conv"):
                    _fill_normal_(p, 0.3, g)
                    p[:, -1] += 1.0
                elif init == "stable" and name.endswith(("norm1.weight", "norm2.weight")):
                    p.fill_(0.05)
                elif "norm" in name:
                    p.fill_(1.0)
                elif leaf == "bias":
                    p.zero_()
                elif init == "stable" and name.endswith(("embed_tokens.weight", "lm_head.weight")):
                    _fill_normal_(p, 1.0, torch.Generator(device="cpu").manual_seed(seed))
                else:
                    _fill_normal_(p, std, g)
            for l in m.model.layers:
                if l.mlp is not None:
                    order = torch.rand(cfg.vocab_size, l.mlp.cfg.experts, generator=g).argsort(-1)
                    l.mlp.table.copy_(order[:, :l.mlp.cfg.top].to(torch.int32))
        return m.eval()

    @classmethod
    def from_pretrained(cls, path: str, dtype=torch.bfloat16, device="cpu") -> "ZasipelForCausalLM":
        from .loader import load_state_into
        m = cls._empty(ZasipelConfig.from_pretrained(path), dtype, device)
        load_state_into(m, path, remap=checkpoint_to_parameter)
        m.check_tables()
        return m.eval()

    def check_tables(self) -> None:
        """Expert tables index expert weights on the device: entries outside the range are refused here."""
        for i, l in enumerate(self.model.layers):
            if l.mlp is not None and not bool(((l.mlp.table >= 0) & (l.mlp.table < l.mlp.cfg.experts)).all()):
                raise ValueError(f"layer {i}: the expert table names experts outside 0 .. {l.mlp.cfg.experts - 1}")

    def save_pretrained(self, path: str) -> None:
        from .loader import save_state
        self.config.save_pretrained(path)
        params = self.state_dict()
        sd = {k: params[v] for k, v in _TOP_NAMES.items()}
        for i, layer in enumerate(self.config.layers):
            base = f"model.layers.{i}."
            sd.update({f"l{i}.{k}": params[base + v] for k, v in _LAYER_NAMES.items() if base + v in params})
            if layer.moe is not None:
                for e in range(layer.moe.experts):
                    sd.update({f"l{i}.mlp.e{e}.{n}": params[f"{base}mlp.w_{n}"][e] for n in _EXPERT_PARTS})
        save_state(sd, path)

    # -- forward ----------------------------------------------------------------
    @torch.inference_mode()
    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor, attn, tap_layers: Optional[Sequence[int]] = None,
                logits_rows=None, router_logits_fn=None, return_hidden: bool = False):
        """Run the decoder on ``input_ids (T,)``.

        ``attn.window(layer, mixer, q, k, v)`` stores K/V rows and attends over the window; ``attn.delta(layer, mixer,
        pre, z, b)`` advances the layer's recurrent states.  The last tapped layer is tapped after the final norm.
        Returns ``(logits, taps or None)``."""
        dtype = self.model.embed_tokens.weight.dtype
        x = self.model.embed_tokens.weight[input_ids].float()
        tap_ids = list(tap_layers) if tap_layers is not None else None
        tapped, last = {}, len(self.model.layers) - 1
        for i, layer in enumerate(self.model.layers):
            recur = lambda pre, z, b, i=i, m=layer.delta: attn.delta(i, m, pre, z, b)
            h = x.to(dtype)
            if isinstance(layer.mixer, SideBySide):
                y = layer.mixer(h, positions, lambda q, k, v, i=i, m=layer.mixer.left: attn.window(i, m, q, k, v), recur)
            else:
                y = layer.mixer(h, recur).float()
            x = x + layer.norm1(y)
            if layer.mlp is not None:
                x = x + layer.norm2(layer.mlp(x.to(dtype), input_ids))
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


register_family("zasipel", ZasipelConfig, ZasipelForCausalLM, aliases=("Zasipel", "ZasipelForCausalLM"))
