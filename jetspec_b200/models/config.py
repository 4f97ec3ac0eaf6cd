"""Model configurations read from ``config.json``: Qwen3 (Hugging Face layout), Karuzen, Zasipel, Kizezen and Sogidra.

Only the fields the decoder actually uses are kept.  The draft head adds
``block_size``, ``num_target_layers`` and ``dflash_config`` on top of the Qwen3
fields (reference: ``jetspec/models/draft_head.py:317-337``).

What the engines, the cache and the kernel path ask of a configuration, whatever the family: ``vocab_size``,
``hidden_size``, ``num_hidden_layers`` (layer RUNS, i.e. cache layers), ``eos_token_id``, ``logit_scale``,
``kernel_path_ok()``, ``kernel_stack()`` (which fused launch sequence runs the decoder, ``None`` for Qwen3's) and what a cache
layer holds: ``latent_widths()`` (width of a latent row, ``None`` where a layer caches none, or ``None`` for a model without),
``kv_shapes()`` (likewise; ``None`` when all layers hold the same K and V heads) and ``state_shapes()`` (``None`` without
recurrent layers).  Optional, for caches of K and V heads: ``kv_sources()`` (per layer, the layer whose keys and values it
reads) and ``kv_pools()`` (per layer, tokens to a pooled block, 0 without).  A model whose positions are a learned table has
``max_positions``.
"""
from __future__ import annotations

import json
import os
from dataclasses import dataclass, field, asdict
from typing import Any, Optional

from .rotary import BandScaling, RampScaling, RotaryConfig


@dataclass
class Qwen3Config:
    vocab_size: int = 151936
    hidden_size: int = 4096
    intermediate_size: int = 12288
    num_hidden_layers: int = 36
    num_attention_heads: int = 32
    num_key_value_heads: int = 8
    head_dim: Optional[int] = 128
    rms_norm_eps: float = 1e-6
    rope_theta: float = 1e6
    max_position_embeddings: int = 40960
    tie_word_embeddings: bool = False
    attention_bias: bool = False
    sliding_window: Optional[int] = None
    layer_types: Optional[list] = None
    eos_token_id: Any = None
    # mixture-of-experts (Qwen3-MoE); num_experts == 0 means a dense model
    num_experts: int = 0
    num_experts_per_tok: int = 0
    moe_intermediate_size: int = 0
    norm_topk_prob: bool = True
    decoder_sparse_step: int = 1
    mlp_only_layers: list = field(default_factory=list)
    # draft-head extras
    block_size: Optional[int] = None
    num_target_layers: Optional[int] = None
    dflash_config: Optional[dict] = None
    model_type: str = "qwen3"

    def __post_init__(self):
        if self.head_dim is None:
            self.head_dim = self.hidden_size // self.num_attention_heads
        if self.layer_types is None:
            self.layer_types = ["full_attention"] * self.num_hidden_layers

    # -- derived sizes ------------------------------------------------------
    @property
    def q_size(self) -> int:
        return self.num_attention_heads * self.head_dim

    @property
    def kv_size(self) -> int:
        return self.num_key_value_heads * self.head_dim

    @property
    def is_moe(self) -> bool:
        return self.num_experts > 0

    def layer_is_moe(self, layer_idx: int) -> bool:
        if not self.is_moe or layer_idx in self.mlp_only_layers:
            return False
        return (layer_idx + 1) % max(1, self.decoder_sparse_step) == 0

    def latent_widths(self) -> Optional[list]:
        """Widths of the latent rows a cache layer holds, or ``None`` when it holds K and V heads."""
        return None

    def kv_shapes(self) -> Optional[list]:
        """Per layer ``(kv_heads, dim, vdim)`` or ``None`` (nothing cached), when layers differ; else ``None``."""
        return None

    def state_shapes(self) -> Optional[list]:
        """Per layer the :class:`DeltaConfig` whose state a sequence carries, or ``None``; ``None`` without any."""
        return None

    logit_scale = 1.0

    def kernel_path_ok(self) -> bool:
        """Whether the graph-captured kernel path covers this geometry."""
        return self.head_dim == 128

    def kernel_stack(self) -> Optional[str]:
        """Name of the fused launch sequence of the decoder (see ``engine.fast_round``); ``None``: ``decoder_layers``."""
        return None

    # -- io -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "Qwen3Config":
        names = set(cls.__dataclass_fields__)
        kw = {k: v for k, v in d.items() if k in names}
        rope = d.get("rope_parameters") or {}
        if "rope_theta" not in kw and "rope_theta" in rope:
            kw["rope_theta"] = rope["rope_theta"]
        return cls(**kw)

    @classmethod
    def from_pretrained(cls, path: str, subfolder: str = "") -> "Qwen3Config":
        p = os.path.join(path, subfolder, "config.json") if subfolder else os.path.join(path, "config.json")
        with open(p) as f:
            d = json.load(f)
        cfg = cls.from_dict(d)
        gen = os.path.join(os.path.dirname(p), "generation_config.json")
        if os.path.exists(gen):
            with open(gen) as f:
                g = json.load(f)
            if g.get("eos_token_id") is not None:
                cfg.eos_token_id = _merge_eos(cfg.eos_token_id, g["eos_token_id"])
        return cfg

    def to_dict(self) -> dict:
        d = asdict(self)
        d["architectures"] = ["Qwen3MoeForCausalLM" if self.is_moe else "Qwen3ForCausalLM"]
        return d

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)


def _as_list(x) -> list:
    if x is None:
        return []
    if isinstance(x, (list, tuple)):
        return [int(v) for v in x]
    return [int(x)]


def _merge_eos(a, b) -> list:
    out = []
    for v in _as_list(a) + _as_list(b):
        if v not in out:
            out.append(v)
    return out


@dataclass
class LatentAttentionConfig:
    """Sizes of a latent attention: queries through a latent of ``q_rank`` (0: one projection), keys and values from one of
    ``kv_rank``; with ``rot`` every query head and the cached row carry ``rot.dims`` rotated entries more."""
    heads: int
    dim: int
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot: Optional[RotaryConfig] = None
    sink_logits: bool = False        # a learned number per head in the softmax's denominator
    gate: bool = False               # sigmoid gate per head on the output

    @property
    def rot_dim(self) -> int:
        return self.rot.dims if self.rot is not None else 0

    @property
    def row(self) -> int:
        """Entries of a cached row: the latent and the rotated key part all heads share."""
        return self.kv_rank + self.rot_dim


@dataclass
class RoutedExpertsConfig:
    """Sizes of a sigmoid-routed expert layer; ``shared_ff`` is 0 without a shared expert."""
    experts: int
    top: int
    scale: float
    ff: int
    shared_ff: int = 0


@dataclass
class KaruzenLayerConfig:
    mixer: LatentAttentionConfig
    dense_ff: int = 0                               # > 0: a dense feed-forward of this width
    moe: Optional[RoutedExpertsConfig] = None       # a layer with neither has no feed-forward


@dataclass
class KaruzenConfig:
    """Karuzen: parallel blocks (latent attention beside a dense or routed feed-forward) under one Dynamic Tanh norm
    each, a range of layers run several times with shared weights, tied embeddings."""
    vocab_size: int
    hidden_size: int
    layers: list
    loop_start: int = 0
    loop_stop: int = 0
    loop_times: int = 1
    norm_eps: float = 1e-5
    eos_token_id: Any = None
    model_type: str = "karuzen"
    logit_scale = 1.0                               # not a field: fixed by the design

    def layer_runs(self) -> list:
        """``[(layer index, add the embedding output before it), ...]`` in execution order.  Every run has its own
        cache layer; the layers of the loop appear once per pass."""
        n, a, b = len(self.layers), self.loop_start, self.loop_stop
        if b <= a:
            return [(i, False) for i in range(n)]
        runs = [(i, False) for i in range(a)]
        for times in range(self.loop_times):
            runs += [(i, times > 0 and i == a) for i in range(a, b)]
        return runs + [(i, False) for i in range(b, n)]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layer_runs())

    @property
    def is_moe(self) -> bool:
        return any(l.moe is not None for l in self.layers)

    def latent_widths(self) -> list:
        return [self.layers[i].mixer.kv_rank for i, _ in self.layer_runs()]

    def kv_shapes(self) -> None:
        return None

    def state_shapes(self) -> None:
        return None

    def kernel_path_ok(self) -> bool:
        return all(l.moe is None or (l.moe.experts <= 1024 and l.moe.top <= 32) for l in self.layers)

    def kernel_stack(self) -> str:
        return "latent"

    # -- io -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "KaruzenConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            m, f = e["mixer"], e.get("mlp")
            lc = KaruzenLayerConfig(LatentAttentionConfig(
                heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]), q_rank=int(m["q_rank"]),
                kv_rank=int(m["kv_rank"]), scale=float(m["scale"])))
            if f is not None and f["kind"] == "dense":
                lc.dense_ff = int(f["ff"])
            elif f is not None and f["kind"] == "moe":
                r, sh = f["router"], f.get("shared")
                lc.moe = RoutedExpertsConfig(experts=int(r["experts"]), top=int(r["top"]), scale=float(r["scale"]),
                                             ff=int(f["expert"]["ff"]), shared_ff=int(sh["ff"]) if sh else 0)
            elif f is not None:
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(lc)
        loop = d.get("loop") or {}
        cfg = cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                  loop_start=int(loop.get("start", 0)), loop_stop=int(loop.get("stop", 0)),
                  loop_times=int(loop.get("times", 1)), norm_eps=float(d["norm"]["eps"]),
                  eos_token_id=d.get("eos_token_id"))
        if not 0 <= cfg.loop_start <= max(cfg.loop_start, cfg.loop_stop) <= len(layers):
            raise ValueError(f"loop {loop} does not fit {len(layers)} layers")
        return cfg

    @classmethod
    def from_pretrained(cls, path: str, subfolder: str = "") -> "KaruzenConfig":
        with open(os.path.join(path, subfolder, "config.json") if subfolder else os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            mlp = None
            if l.dense_ff:
                mlp = {"kind": "dense", "ff": l.dense_ff}
            elif l.moe is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.moe.ff},
                       "router": {"experts": l.moe.experts, "top": l.moe.top, "scale": l.moe.scale}}
                if l.moe.shared_ff:
                    mlp["shared"] = {"ff": l.moe.shared_ff}
            m = l.mixer
            layers.append({"type": "latent_attention", "mlp": mlp, "mixer": {
                "heads": m.heads, "dim": m.dim, "vdim": m.vdim, "q_rank": m.q_rank, "kv_rank": m.kv_rank, "scale": m.scale}})
        d = {"architecture": "Karuzen", "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
             "norm": {"eps": self.norm_eps}}
        if self.loop_stop > self.loop_start:
            d["loop"] = {"start": self.loop_start, "stop": self.loop_stop, "times": self.loop_times}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)



@dataclass
class WindowAttentionConfig:
    """Sizes and constants of an attention over grouped K/V heads, in a sliding window or over the whole past: a token sees
    itself and the ``window - 1`` tokens before it (``window`` 0: all of them), the sequence's first ``keep_first`` tokens, and
    with ``pool`` one key and value for each whole block of that many tokens behind the window, the means over the block.
    The first ``rot_dims`` dimensions are rotated in neighbouring pairs, or as ``rot`` says."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    window: int
    rot_dims: int
    rot_base: float
    scale: float
    sink: bool = True                # a valueless key of score 0 takes part in the softmax
    qk_norm: bool = True             # weightless RMS norm of q and k behind the rotation
    bias: bool = True                # biases on all four projections
    keep_first: int = 0
    sink_logits: bool = False        # a learned number per head in the softmax's denominator (instead of ``sink``)
    proj_norm: bool = False          # weighted RMS norm over the whole q and k projections ahead of the rotation
    o_bias: Optional[bool] = None    # bias on the output projection; None: as ``bias``
    gate: bool = False               # sigmoid gate per head on the output
    rot: Optional[RotaryConfig] = None
    pool: int = 0
    softcap: float = 0.0             # > 0: scores pass through softcap * tanh(score / softcap)
    tie_values: bool = False         # the values are the keys as projected, ahead of norm and rotation
    diff: Optional[float] = None     # differential attention: two maps a head over the same values, a1 - lambda a2 normed
    temp_every: int = 0              # > 0: q is multiplied by 1 + temp_coef ln(floor((p + 1) / temp_every) + 1)
    temp_coef: float = 0.0
    kv_from: Optional[int] = None    # no keys and values of its own: those of this layer

    @property
    def maps(self) -> int:
        """Attention maps of a head; q and k carry one vector for each."""
        return 2 if self.diff is not None else 1


@dataclass
class DeltaConfig:
    """Sizes of a gated delta rule.  ``decay``: one per ``"head"`` or per ``"channel"`` of the key; ``gate``: activation
    of the output gate.  A rank of 0 makes that projection a single matrix, else it goes through that rank."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    taps: int
    decay: str = "head"
    gate: str = "silu"
    decay_rank: int = 0
    gate_rank: int = 0

    @property
    def held(self) -> list:
        """``(width, fp32?)`` of the rows that enter the recurrence (see ``GatedDelta.mix``)."""
        return [(self.channels, False), (self.decays, True), (self.heads, True)]

    @property
    def channels(self) -> int:
        """Channels of the short convolution: q, k and v side by side."""
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def decays(self) -> int:
        return self.heads * (self.dim if self.decay == "channel" else 1)


@dataclass
class TableExpertsConfig:
    """Experts a table of token ids names, with equal weights; ``shared_ff`` is 0 without a shared expert."""
    experts: int
    top: int
    ff: int
    shared_ff: int = 0


@dataclass
class ZasipelLayerConfig:
    """``window`` beside ``delta`` (a parallel layer), or ``delta`` alone."""
    delta: DeltaConfig
    window: Optional[WindowAttentionConfig] = None
    moe: Optional[TableExpertsConfig] = None        # None: no feed-forward

    @property
    def mixer_type(self) -> str:
        return "parallel" if self.window is not None else "channel_delta"


@dataclass
class ZasipelConfig:
    """Zasipel: window attention and a gated delta rule side by side, or a channel-decay delta rule alone; experts chosen
    by token id; norms on the sublayers' outputs only; untied head."""
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float = 1e-6
    eos_token_id: Any = None
    model_type: str = "zasipel"
    logit_scale = 1.0                               # not a field: fixed by the design

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def is_moe(self) -> bool:
        return any(l.moe is not None for l in self.layers)

    def latent_widths(self) -> None:
        return None

    def kv_shapes(self) -> list:
        return [(l.window.kv_heads, l.window.dim, l.window.vdim) if l.window is not None else None for l in self.layers]

    def state_shapes(self) -> list:
        return [l.delta for l in self.layers]

    def kernel_path_ok(self) -> bool:
        return all(l.delta.dim <= 256 and l.delta.vdim <= 256 and l.delta.taps <= 17
                   and (l.window is None or (l.window.dim <= 512 and l.window.vdim <= 512))
                   and (l.moe is None or l.moe.experts <= 1024) for l in self.layers)

    def kernel_stack(self) -> str:
        return "hybrid"

    # -- io -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict, shape_of=None) -> "ZasipelConfig":
        """``shape_of(tensor name)`` gives the two low ranks of a channel-decay layer, which only the weights tell
        (without it: a quarter of the head size)."""
        def delta(m, p, decay):
            c = DeltaConfig(heads=int(m["heads"]), kv_heads=int(m["kv_heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]),
                            taps=int(m["conv"]), decay=decay, gate="silu" if decay == "head" else "sigmoid")
            if decay == "channel":
                rank = lambda n, e: int(shape_of(p + n)[0]) if shape_of is not None else max(1, e // 4)
                c.decay_rank, c.gate_rank = rank(".a1", c.dim), rank(".g1", c.vdim)
            return c

        layers = []
        for i, e in enumerate(d["layers"]):
            m, f, p = e["mixer"], e.get("mlp"), f"l{i}.mix"
            if e["type"] == "parallel":
                a = m["left"]
                lc = ZasipelLayerConfig(delta(m["right"], p + ".right", "head"), window=WindowAttentionConfig(
                    heads=int(a["heads"]), kv_heads=int(a["kv_heads"]), dim=int(a["dim"]), vdim=int(a["vdim"]),
                    window=int(a["mask"]["size"]), rot_dims=int(a["rot"]["dims"]), rot_base=float(a["rot"]["base"]),
                    scale=float(a["scale"])))
            elif e["type"] == "channel_delta":
                lc = ZasipelLayerConfig(delta(m, p, "channel"))
            else:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            for c in (lc.delta, lc.window):
                if c is not None and c.heads % c.kv_heads:
                    raise ValueError(f"layer {i}: {c.heads} heads do not divide over {c.kv_heads} key heads")
            if f is not None:
                if f["kind"] != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
                r, sh = f["router"], f.get("shared")
                lc.moe = TableExpertsConfig(experts=int(r["experts"]), top=int(r["top"]), ff=int(f["expert"]["ff"]),
                                            shared_ff=int(sh["ff"]) if sh else 0)
            layers.append(lc)
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers,
                   norm_eps=float(d["norm"]["eps"]), eos_token_id=d.get("eos_token_id"))

    @classmethod
    def from_pretrained(cls, path: str, subfolder: str = "") -> "ZasipelConfig":
        from .loader import tensor_shape
        base = os.path.join(path, subfolder) if subfolder else path
        with open(os.path.join(base, "config.json")) as f:
            return cls.from_dict(json.load(f), shape_of=lambda name: tensor_shape(base, name))

    def to_dict(self) -> dict:
        def delta(c):
            return {"heads": c.heads, "kv_heads": c.kv_heads, "dim": c.dim, "vdim": c.vdim, "conv": c.taps}

        layers = []
        for l in self.layers:
            mixer = delta(l.delta)
            if l.window is not None:
                a = l.window
                mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                                  "mask": {"size": a.window}, "rot": {"dims": a.rot_dims, "base": a.rot_base}},
                         "right": mixer}
            mlp = None
            if l.moe is not None:
                mlp = {"kind": "moe", "expert": {"ff": l.moe.ff}, "router": {"experts": l.moe.experts, "top": l.moe.top}}
                if l.moe.shared_ff:
                    mlp["shared"] = {"ff": l.moe.shared_ff}
            layers.append({"type": l.mixer_type, "mixer": mixer, "mlp": mlp})
        d = {"architecture": "Zasipel", "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
             "norm": {"eps": self.norm_eps}}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)


@dataclass
class RetentionConfig:
    """Sizes of a retention: linear attention with one fixed decay per head and rotated queries and keys."""
    heads: int
    dim: int
    vdim: int
    decay: list
    rot: RotaryConfig
    taps = channels = 0              # no short convolution: a sequence carries the state alone

    @property
    def held(self) -> list:
        """``(width, fp32?)`` of the rows that enter the recurrence (see ``Retention.mix``)."""
        return [(self.heads * self.dim, True), (self.heads * self.dim, True), (self.heads * self.vdim, False)]


@dataclass
class KizezenLayerConfig:
    """``mixer``: a :class:`WindowAttentionConfig`, :class:`LatentAttentionConfig` or :class:`RetentionConfig`."""
    mixer: Any
    ff: int = 0                      # width of the feed-forward, 0 without one

    @property
    def mixer_type(self) -> str:
        return {WindowAttentionConfig: "attention", LatentAttentionConfig: "latent_attention", RetentionConfig: "retention"}[type(self.mixer)]


@dataclass
class KizezenConfig:
    """Kizezen: pre-norm blocks whose mixers are window attention, latent attention or retention, in any order; scaled
    embeddings and logits; untied head."""
    vocab_size: int
    hidden_size: int
    layers: list
    norm_eps: float = 1e-5
    embed_scale: float = 1.0
    logit_scale: float = 1.0
    eos_token_id: Any = None
    model_type: str = "kizezen"
    is_moe = False

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def _per_layer(self, kind, of) -> Optional[list]:
        out = [of(l.mixer) if isinstance(l.mixer, kind) else None for l in self.layers]
        return out if any(x is not None for x in out) else None

    def latent_widths(self) -> Optional[list]:
        return self._per_layer(LatentAttentionConfig, lambda m: m.row)

    def kv_shapes(self) -> list:
        return self._per_layer(WindowAttentionConfig, lambda m: (m.kv_heads, m.dim, m.vdim)) or [None] * len(self.layers)

    def state_shapes(self) -> Optional[list]:
        return self._per_layer(RetentionConfig, lambda m: m)

    def kernel_path_ok(self) -> bool:
        """Sizes the fused kernels take, and a logit scale that keeps the order of the logits."""
        def ok(m):
            if isinstance(m, WindowAttentionConfig):
                return m.dim <= 512 and m.vdim <= 512
            return m.row <= 2048 if isinstance(m, LatentAttentionConfig) else m.dim <= 256
        return self.logit_scale > 0 and all(ok(l.mixer) for l in self.layers)

    def kernel_stack(self) -> str:
        return "prenorm"

    # -- io -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "KizezenConfig":
        def band(s):
            return None if s is None else BandScaling(*(float(s[k]) for k in ("factor", "low", "high", "original")))

        def ramp(s):
            return None if s is None else RampScaling(*(float(s[k]) for k in ("factor", "original", "fast", "slow")))

        def mixer(i, t, m):
            r, size = m["rot"], {k: int(m[k]) for k in ("heads", "dim", "vdim")}
            dims, base = int(r["dims"]), float(r["base"])
            if t == "attention":
                if size["heads"] % int(m["kv_heads"]):
                    raise ValueError(f"layer {i}: {m['heads']} heads do not divide over {m['kv_heads']} key heads")
                return WindowAttentionConfig(
                    **size, kv_heads=int(m["kv_heads"]), window=int(m["mask"]["size"]), keep_first=int(m["mask"]["keep_first"]),
                    rot_dims=dims, rot_base=base, rot=RotaryConfig(dims, base, "half", band(r.get("scaling"))), scale=float(m["scale"]),
                    sink=False, sink_logits=True, qk_norm=False, proj_norm=True, bias=True, o_bias=False, gate=True)
            if t == "latent_attention":
                if dims != int(m["rot_dim"]):
                    raise ValueError(f"layer {i}: {dims} rotated entries, but rot_dim {m['rot_dim']}")
                return LatentAttentionConfig(**size, q_rank=0, kv_rank=int(m["kv_rank"]), scale=float(m["scale"]),
                                             rot=RotaryConfig(dims, base, "next", ramp(r.get("scaling"))), sink_logits=True, gate=True)
            if t == "retention":
                decay = [float(x) for x in m["decay"]]
                if len(decay) != size["heads"]:
                    raise ValueError(f"layer {i}: {len(decay)} decays for {size['heads']} heads")
                return RetentionConfig(**size, decay=decay, rot=RotaryConfig(dims, base, "half"))
            raise ValueError(f"layer {i}: unknown mixer type {t!r}")

        layers = []
        for i, e in enumerate(d["layers"]):
            f = e.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            lc = KizezenLayerConfig(mixer(i, e["type"], e["mixer"]), ff=int(f["ff"]) if f is not None else 0)
            if lc.mixer_type != "latent_attention" and lc.mixer.rot.dims > lc.mixer.dim:
                raise ValueError(f"layer {i}: {lc.mixer.rot.dims} rotated entries in heads of {lc.mixer.dim}")
            layers.append(lc)
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, norm_eps=float(d["norm"]["eps"]),
                   embed_scale=float(d["embedding"]["scale"]), logit_scale=float(d["logit_scale"]), eos_token_id=d.get("eos_token_id"))

    @classmethod
    def from_pretrained(cls, path: str, subfolder: str = "") -> "KizezenConfig":
        with open(os.path.join(path, subfolder, "config.json") if subfolder else os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m, r = l.mixer, l.mixer.rot
            mixer = {"heads": m.heads, "dim": m.dim, "vdim": m.vdim, "rot": {"dims": r.dims, "base": r.base}}
            if r.scaling is not None:
                mixer["rot"]["scaling"] = asdict(r.scaling)
            if isinstance(m, WindowAttentionConfig):
                mixer.update(kv_heads=m.kv_heads, scale=m.scale, mask={"size": m.window, "keep_first": m.keep_first})
            elif isinstance(m, LatentAttentionConfig):
                mixer.update(kv_rank=m.kv_rank, rot_dim=m.rot_dim, scale=m.scale)
            else:
                mixer["decay"] = list(m.decay)
            layers.append({"type": l.mixer_type, "mixer": mixer, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        d = {"architecture": "Kizezen", "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
             "norm": {"eps": self.norm_eps}, "embedding": {"scale": self.embed_scale}, "logit_scale": self.logit_scale}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)


@dataclass
class SogidraLayerConfig:
    mixer: WindowAttentionConfig
    ff: int = 0                      # width of the feed-forward, 0 without one

    @property
    def mixer_type(self) -> str:
        return "attention" if self.mixer.diff is not None else "attention_2"


@dataclass
class SogidraConfig:
    """Sogidra: differential attention over the whole past and window attention with pooled blocks, in any order, keys and
    values shared between layers; norms before and after every sublayer; a weighted average over the depth behind every layer;
    learned positions; tied head."""
    vocab_size: int
    hidden_size: int
    layers: list
    max_positions: int
    norm_eps: float = 1e-6
    eos_token_id: Any = None
    model_type: str = "sogidra"
    logit_scale = embed_scale = 1.0                 # not fields: fixed by the design
    is_moe = False

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    def latent_widths(self) -> None:
        return None

    def kv_shapes(self) -> list:
        return [(m.kv_heads, m.dim, m.vdim, m.maps) if m.kv_from is None else None for m in (l.mixer for l in self.layers)]

    def kv_sources(self) -> list:
        return [i if l.mixer.kv_from is None else l.mixer.kv_from for i, l in enumerate(self.layers)]

    def kv_pools(self) -> list:
        return [l.mixer.pool for l in self.layers]

    def state_shapes(self) -> None:
        return None

    def kernel_path_ok(self) -> bool:
        return self.hidden_size <= 32768 and all(l.mixer.dim <= 512 and l.mixer.vdim <= 512 for l in self.layers)

    def kernel_stack(self) -> str:
        return "prenorm"

    # -- io -------------------------------------------------------------------
    @classmethod
    def from_dict(cls, d: dict) -> "SogidraConfig":
        def mixer(i, t, m):
            size = {k: int(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")}
            if size["heads"] % size["kv_heads"]:
                raise ValueError(f"layer {i}: {m['heads']} heads do not divide over {m['kv_heads']} key heads")
            common = dict(**size, scale=float(m["scale"]), rot_dims=0, rot_base=1.0, sink=False, o_bias=False)
            if t == "attention":
                temp, src = m.get("q_temp") or {}, m.get("kv_from")
                return WindowAttentionConfig(**common, window=0, qk_norm=False, bias=True, diff=float(m["diff"]),
                                             temp_every=int(temp.get("every", 0)), temp_coef=float(temp.get("coef", 0.0)),
                                             kv_from=int(src) if src is not None else None)
            if t == "attention_2":
                if size["dim"] != size["vdim"]:
                    raise ValueError(f"layer {i}: values are keys, but heads have {m['dim']} and {m['vdim']} entries")
                if int(m["mask"]["size"]) < 1 or int(m["mask"]["pool"]) < 1:
                    raise ValueError(f"layer {i}: mask {m['mask']}")
                return WindowAttentionConfig(**common, window=int(m["mask"]["size"]), pool=int(m["mask"]["pool"]), qk_norm=True, bias=False,
                                             tie_values=True, softcap=float(m["softcap"]))
            raise ValueError(f"layer {i}: unknown mixer type {t!r}")

        layers = []
        for i, e in enumerate(d["layers"]):
            f = e.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward kind {f['kind']!r}")
            layers.append(SogidraLayerConfig(mixer(i, e["type"], e["mixer"]), ff=int(f["ff"]) if f is not None else 0))
        for i, l in enumerate(layers):
            m = l.mixer
            if m.kv_from is None:
                continue
            src = layers[m.kv_from].mixer if 0 <= m.kv_from < i else None
            if src is None or src.diff is None or src.kv_from is not None or (src.kv_heads, src.dim, src.vdim) != (m.kv_heads, m.dim, m.vdim):
                raise ValueError(f"layer {i} cannot use the keys and values of layer {m.kv_from}")
        return cls(vocab_size=int(d["vocab"]), hidden_size=int(d["width"]), layers=layers, max_positions=int(d["max_positions"]),
                   norm_eps=float(d["norm"]["eps"]), eos_token_id=d.get("eos_token_id"))

    @classmethod
    def from_pretrained(cls, path: str, subfolder: str = "") -> "SogidraConfig":
        with open(os.path.join(path, subfolder, "config.json") if subfolder else os.path.join(path, "config.json")) as f:
            return cls.from_dict(json.load(f))

    def to_dict(self) -> dict:
        layers = []
        for l in self.layers:
            m = l.mixer
            mixer = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.vdim, "scale": m.scale}
            if m.diff is not None:
                mixer["diff"] = m.diff
                if m.temp_every:
                    mixer["q_temp"] = {"every": m.temp_every, "coef": m.temp_coef}
                if m.kv_from is not None:
                    mixer["kv_from"] = m.kv_from
            else:
                mixer.update(softcap=m.softcap, mask={"size": m.window, "pool": m.pool})
            layers.append({"type": l.mixer_type, "mixer": mixer, "mlp": {"kind": "dense", "ff": l.ff} if l.ff else None})
        d = {"architecture": "Sogidra", "vocab": self.vocab_size, "width": self.hidden_size, "layers": layers,
             "norm": {"eps": self.norm_eps}, "max_positions": self.max_positions}
        if self.eos_token_id is not None:
            d["eos_token_id"] = self.eos_token_id
        return d

    def save_pretrained(self, path: str) -> None:
        os.makedirs(path, exist_ok=True)
        with open(os.path.join(path, "config.json"), "w") as f:
            json.dump(self.to_dict(), f, indent=1)


# Geometry presets used by the tests and the benchmarks (random-init weights).
def tiny_config(**over) -> Qwen3Config:
    """2 layers, hidden 256, 4 q / 2 kv heads, head_dim 64, SwiGLU 512, vocab 1024."""
    kw = dict(vocab_size=1024, hidden_size=256, intermediate_size=512, num_hidden_layers=2,
              num_attention_heads=4, num_key_value_heads=2, head_dim=64, rope_theta=1e6,
              rms_norm_eps=1e-6, max_position_embeddings=4096)
    kw.update(over)
    return Qwen3Config(**kw)


def qwen3_8b_config(**over) -> Qwen3Config:
    kw = dict(vocab_size=151936, hidden_size=4096, intermediate_size=12288, num_hidden_layers=36,
              num_attention_heads=32, num_key_value_heads=8, head_dim=128, rope_theta=1e6)
    kw.update(over)
    return Qwen3Config(**kw)


def qwen3_30b_a3b_config(**over) -> Qwen3Config:
    kw = dict(vocab_size=151936, hidden_size=2048, intermediate_size=6144, num_hidden_layers=48,
              num_attention_heads=32, num_key_value_heads=4, head_dim=128, rope_theta=1e6,
              num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768,
              norm_topk_prob=True, model_type="qwen3_moe")
    kw.update(over)
    return Qwen3Config(**kw)


def karuzen_tiny_config(**over) -> KaruzenConfig:
    """4 layers (dense, routed, routed, no feed-forward), the middle two run three times; width 192, 3 heads."""
    mix = LatentAttentionConfig(heads=3, dim=40, vdim=24, q_rank=56, kv_rank=72, scale=0.2)
    moe = RoutedExpertsConfig(experts=6, top=2, scale=1.3, ff=48, shared_ff=80)
    kw = dict(vocab_size=320, hidden_size=192, norm_eps=1e-5, loop_start=1, loop_stop=3, loop_times=3,
              layers=[KaruzenLayerConfig(mix, dense_ff=160), KaruzenLayerConfig(mix, moe=moe),
                      KaruzenLayerConfig(mix, moe=moe), KaruzenLayerConfig(mix)])
    kw.update(over)
    return KaruzenConfig(**kw)


def karuzen_bench_config(layers: int = 16, moe: bool = False, **over) -> KaruzenConfig:
    """Width 4096, 32 heads of 128, latents of 1536 and 512, feed-forward 12288 (or 64 experts of 1536, 8 a token)."""
    mix = LatentAttentionConfig(heads=32, dim=128, vdim=128, q_rank=1536, kv_rank=512, scale=128 ** -0.5)
    ex = RoutedExpertsConfig(experts=64, top=8, scale=2.5, ff=1536, shared_ff=1536)
    kw = dict(vocab_size=151936, hidden_size=4096, layers=[
        KaruzenLayerConfig(mix, moe=ex) if moe else KaruzenLayerConfig(mix, dense_ff=12288) for _ in range(layers)])
    kw.update(over)
    return KaruzenConfig(**kw)


def zasipel_tiny_config(**over) -> ZasipelConfig:
    """3 layers (parallel, channel decay, parallel without a feed-forward); width 160."""
    win = WindowAttentionConfig(heads=6, kv_heads=2, dim=24, vdim=40, window=21, rot_dims=12, rot_base=1e4, scale=0.3)
    head = DeltaConfig(heads=4, kv_heads=2, dim=16, vdim=32, taps=4)
    chan = DeltaConfig(heads=3, kv_heads=3, dim=24, vdim=16, taps=4, decay="channel", gate="sigmoid", decay_rank=10, gate_rank=6)
    moe = TableExpertsConfig(experts=6, top=3, ff=40, shared_ff=56)
    kw = dict(vocab_size=320, hidden_size=160, norm_eps=1e-5,
              layers=[ZasipelLayerConfig(head, win, moe), ZasipelLayerConfig(chan, None, moe), ZasipelLayerConfig(head, win, None)])
    kw.update(over)
    return ZasipelConfig(**kw)


def kizezen_tiny_config(**over) -> KizezenConfig:
    """4 layers (retention, window attention, latent attention, window attention without a feed-forward); width 144."""
    def win(window, keep, rot):
        return WindowAttentionConfig(heads=6, kv_heads=2, dim=24, vdim=40, window=window, keep_first=keep, rot_dims=rot.dims, rot_base=rot.base,
                                     rot=rot, scale=0.25, sink=False, sink_logits=True, qk_norm=False, proj_norm=True, bias=True,
                                     o_bias=False, gate=True)
    ret = RetentionConfig(heads=3, dim=20, vdim=28, decay=[0.9, 0.97, 0.995], rot=RotaryConfig(12, 1e4))
    lat = LatentAttentionConfig(heads=5, dim=24, vdim=20, q_rank=0, kv_rank=56, scale=0.2, sink_logits=True, gate=True,
                                rot=RotaryConfig(8, 1e4, "next", RampScaling(8.0, 256, 16.0, 2.0)))
    kw = dict(vocab_size=320, hidden_size=144, norm_eps=1e-5, embed_scale=1.5, logit_scale=0.5, layers=[
        KizezenLayerConfig(ret, 168), KizezenLayerConfig(win(21, 3, RotaryConfig(16, 1e4, "half", BandScaling(8.0, 1.0, 4.0, 128))), 200),
        KizezenLayerConfig(lat, 120), KizezenLayerConfig(win(9, 0, RotaryConfig(24, 5e3)))])
    kw.update(over)
    return KizezenConfig(**kw)


def sogidra_tiny_config(**over) -> SogidraConfig:
    """4 layers (pooled window, differential, pooled window without a feed-forward, differential on the second layer's keys);
    width 136."""
    def diff(**kw):
        return WindowAttentionConfig(heads=4, kv_heads=2, dim=20, vdim=36, window=0, rot_dims=0, rot_base=1.0, scale=0.25, sink=False,
                                     qk_norm=False, bias=True, o_bias=False, diff=0.4, temp_every=16, temp_coef=0.3, **kw)

    def pooled(window, pool):
        return WindowAttentionConfig(heads=6, kv_heads=2, dim=28, vdim=28, window=window, rot_dims=0, rot_base=1.0, scale=0.4, sink=False,
                                     qk_norm=True, bias=False, o_bias=False, tie_values=True, softcap=20.0, pool=pool)
    kw = dict(vocab_size=320, hidden_size=136, max_positions=512, norm_eps=1e-5, layers=[
        SogidraLayerConfig(pooled(21, 5), 168), SogidraLayerConfig(diff(), 200), SogidraLayerConfig(pooled(9, 8)),
        SogidraLayerConfig(diff(kv_from=1), 120)])
    kw.update(over)
    return SogidraConfig(**kw)


def draft_head_config(target: Qwen3Config, num_layers: int = 1, block_size: int = 16,
                      target_layer_ids: Optional[list] = None, mask_token_id: Optional[int] = None,
                      num_taps: int = 5, causal_head: bool = True) -> Qwen3Config:
    """Config of a causal-parallel draft head attached to ``target``."""
    from .draft_head import build_target_layer_ids
    ids = target_layer_ids or build_target_layer_ids(target.num_hidden_layers, num_taps)
    if not hasattr(target, "head_dim"):         # the head keeps its own K/V attention: 128-wide heads over the width
        n = max(1, target.hidden_size // 128)
        geometry = dict(intermediate_size=3 * target.hidden_size, num_attention_heads=n, num_key_value_heads=n, head_dim=128,
                        rms_norm_eps=target.norm_eps)
    else:
        geometry = dict(intermediate_size=target.intermediate_size, num_attention_heads=target.num_attention_heads,
                        num_key_value_heads=target.num_key_value_heads, head_dim=target.head_dim,
                        rms_norm_eps=target.rms_norm_eps, rope_theta=target.rope_theta)
    return Qwen3Config(
        vocab_size=target.vocab_size, hidden_size=target.hidden_size, num_hidden_layers=num_layers, **geometry,
        block_size=block_size, num_target_layers=target.num_hidden_layers,
        dflash_config={"causal_head": causal_head, "target_layer_ids": list(ids),
                       "target_hidden_size": target.hidden_size,
                       "mask_token_id": target.vocab_size - 1 if mask_token_id is None else mask_token_id},
    )
