"""Plain, slow statement of the Kizezen design: one function per mechanism, one sequence at a time, no cache.

Written from the equations alone; it shares no code with ``jetspec_b200``.  Everything runs in the dtype of the weights
handed in (float64 in most tests), so it is the yardstick both for the 32-bit and the bf16 product paths.

Notation: ``x`` is the residual stream ``(T, width)``, ``h`` a sublayer's normed input, ``w`` a dict of weight tensors with
the checkpoint's names, linear weights ``(out, in)``; row ``t`` of a matrix belongs to token ``t``.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ pieces
def rms(x, eps):
    """``x`` divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps)


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def gelu(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def plain_freqs(dims, base):
    return [float(base) ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_freqs(dims, base, s):
    """Wavelengths short against ``original / high`` keep their frequency, long against ``original / low`` have it divided by
    ``factor``; linear in ``original / wavelength`` between the two."""
    out = []
    for f in plain_freqs(dims, base):
        wave = 2.0 * math.pi / f
        if wave < s["original"] / s["high"]:
            out.append(f)
        elif wave > s["original"] / s["low"]:
            out.append(f / s["factor"])
        else:
            t = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
            out.append((1.0 - t) * f / s["factor"] + t * f)
    return out


def ramped_freqs(dims, base, s):
    """YaRN: a ramp over the pair index between the pairs that turn ``fast`` and ``slow`` times within ``original`` tokens;
    returns the frequencies and the factor on cosine and sine."""
    at = lambda turns: dims * math.log(s["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))
    lo, hi = max(math.floor(at(s["fast"])), 0), min(math.ceil(at(s["slow"])), dims - 1)
    out = []
    for i, f in enumerate(plain_freqs(dims, base)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / s["factor"] * r + f * (1.0 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, freqs, partner, positions, amp=1.0):
    """Turn the pairs of the first ``2 len(freqs)`` entries of every head, ``x (T, heads, dim)``.  ``partner``: ``"half"``
    pairs entry ``i`` with ``i + n``, ``"next"`` entry ``2i`` with ``2i + 1``."""
    out, n = x.clone(), len(freqs)
    for i, f in enumerate(freqs):
        a, b = (i, i + n) if partner == "half" else (2 * i, 2 * i + 1)
        ang = positions.to(torch.float64) * f
        c, s = (amp * torch.cos(ang)).to(x.dtype)[:, None], (amp * torch.sin(ang)).to(x.dtype)[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a], out[..., b] = u * c - v * s, v * c + u * s
    return out


def softmax_with_sink(s, seen, sink):
    """Weights ``(T, T)`` of scores ``s`` where ``seen``; ``exp(sink)`` is one more term of the denominator."""
    s = s.masked_fill(~seen, -math.inf)
    top = torch.clamp(s.max(-1, keepdim=True).values, min=float(sink)) if sink is not None else s.max(-1, keepdim=True).values
    e = torch.exp(s - top)
    extra = torch.exp(sink - top) if sink is not None else 0.0
    return e / (e.sum(-1, keepdim=True) + extra)


# ------------------------------------------------------------------ mixers
def attention(h, w, p, m, eps, fault=None):
    """Grouped-head attention, norms over whole projections, half rotation, window with kept first tokens, sinks, one gate per
    head.  ``fault`` (tests that plant one): ``"no_sink"``, ``"no_gate"`` or a pair ``(i, j)`` whose visibility is flipped."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rms(h @ w[p + ".q"].T + w[p + ".q.b"], eps) * w[p + ".q.norm"]
    k = rms(h @ w[p + ".k"].T + w[p + ".k.b"], eps) * w[p + ".k.norm"]
    v = (h @ w[p + ".v"].T + w[p + ".v.b"]).view(T, G, V)
    r, pos = m["rot"], torch.arange(T)
    freqs = banded_freqs(r["dims"], r["base"], r["scaling"]) if r.get("scaling") else plain_freqs(r["dims"], r["base"])
    q, k = rotate(q.view(T, H, D), freqs, "half", pos), rotate(k.view(T, G, D), freqs, "half", pos)
    back = pos[:, None] - pos[None]
    seen = (back >= 0) & ((back < m["mask"]["size"]) | (pos[None] < m["mask"]["keep_first"]))
    if isinstance(fault, tuple):
        seen[fault] = ~seen[fault]
    gate = sigmoid(h @ w[p + ".g"].T)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        a = softmax_with_sink(q[:, n] @ k[:, n // (H // G)].T * m["scale"], seen, None if fault == "no_sink" else w[p + ".sink"][n])
        out[:, n] = a @ v[:, n // (H // G)]
        if fault != "no_gate":
            out[:, n] *= gate[:, n, None]
    return out.reshape(T, H * V) @ w[p + ".o"].T


def latent_attention(h, w, p, m, eps, fault=None):
    """Keys and values from a normed latent, a rotated key part shared by the heads, sinks, one gate per head."""
    T, H, D, R, V = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    r, pos = m["rot"], torch.arange(T)
    freqs, amp = ramped_freqs(R, r["base"], r["scaling"]) if r.get("scaling") else (plain_freqs(R, r["base"]), 1.0)
    q = (h @ w[p + ".q"].T).view(T, H, D + R)
    down = h @ w[p + ".dkv"].T
    c = rms(down[:, : m["kv_rank"]], eps) * w[p + ".dkv.norm"]
    qr = rotate(q[..., D:], freqs, "next", pos, amp)
    kr = rotate(down[:, None, m["kv_rank"]:], freqs, "next", pos, amp)[:, 0]
    k, v = (c @ w[p + ".uk"].T).view(T, H, D), (c @ w[p + ".uv"].T).view(T, H, V)
    seen = pos[:, None] >= pos[None]
    if isinstance(fault, tuple):
        seen[fault] = ~seen[fault]
    gate = sigmoid(h @ w[p + ".g"].T)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        s = (q[:, n, :D] @ k[:, n].T + qr[:, n] @ kr.T) * m["scale"]
        out[:, n] = gate[:, n, None] * (softmax_with_sink(s, seen, None if fault == "no_sink" else w[p + ".sink"][n]) @ v[:, n])
    return out.reshape(T, H * V) @ w[p + ".o"].T


def retention_rule(q, k, v, decay, S=None):
    """One head, token by token: ``S <- decay S + k v^T``, read out with ``q``.  Returns read-outs and the last state."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=q.dtype) if S is None else S.clone()
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = decay * S + torch.outer(k[t], v[t])
        out[t] = S.T @ q[t]
    return out, S


def retention(h, w, p, m, eps):
    """Linear attention with one fixed decay per head; per-head norm without a weight, silu gate over all columns."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    freqs, pos = plain_freqs(m["rot"]["dims"], m["rot"]["base"]), torch.arange(T)
    q = rotate((h @ w[p + ".q"].T).view(T, H, D), freqs, "half", pos)
    k = rotate((h @ w[p + ".k"].T).view(T, H, D), freqs, "half", pos) / math.sqrt(D)
    v = (h @ w[p + ".v"].T).view(T, H, V)
    o = torch.stack([retention_rule(q[:, n], k[:, n], v[:, n], m["decay"][n])[0] for n in range(H)], 1)
    return (rms(o, eps).reshape(T, H * V) * silu(h @ w[p + ".g"].T)) @ w[p + ".o"].T


MIXERS = {"attention": attention, "latent_attention": latent_attention, "retention": retention}


# ------------------------------------------------------------------ the decoder
def feed_forward(h, w, p):
    return gelu(h @ w[p + ".up"].T) @ w[p + ".down"].T


def layer(x, w, i, cfg, **fault):
    L, p, eps = cfg["layers"][i], f"l{i}", cfg["norm"]["eps"]
    x = x + MIXERS[L["type"]](rms(x, eps) * w[p + ".norm1"], w, p + ".mix", L["mixer"], eps, **fault)
    if L["mlp"] is not None:
        x = x + feed_forward(rms(x, eps) * w[p + ".norm2"], w, p + ".mlp")
    return x


def forward(tokens, w, cfg, streams=None, faults=None):
    """Logits ``(T, vocab)`` of one whole sequence; ``streams`` collects the residual stream after every layer; ``faults``
    maps a layer to a planted fault of its mixer."""
    x = w["embed"][[int(t) for t in tokens]] * cfg["embedding"]["scale"]
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg, **({"fault": faults[i]} if faults and i in faults else {}))
        if streams is not None:
            streams.append(x)
    return (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T * cfg["logit_scale"]


def greedy(tokens, w, cfg, n):
    """``n`` greedy continuations, recomputing the whole sequence for every token."""
    ids = list(tokens)
    for _ in range(n):
        ids.append(int(forward(ids, w, cfg)[-1].argmax()))
    return ids[len(tokens):]


# ------------------------------------------------------------------ random models for the tests
def random_weights(cfg, seed=0, dtype=torch.float64):
    """Weights of every tensor ``cfg`` implies, rounded to bf16 (what a checkpoint holds)."""
    g = torch.Generator().manual_seed(seed)
    w, W, V = {}, cfg["width"], cfg["vocab"]
    bf = lambda x: x.to(torch.bfloat16).to(dtype)

    def mat(name, *shape, std=None):
        w[name] = bf(torch.randn(*shape, generator=g) * (std if std is not None else 1.0 / math.sqrt(shape[-1])))

    def vec(name, n, around, spread):
        w[name] = bf(around + spread * torch.randn(n, generator=g))

    mat("embed", V, W, std=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", L["mixer"], L["mlp"]
        H, D, E = m["heads"], m["dim"], m["vdim"]
        vec(p + ".norm1", W, 1.0, 0.2)
        if L["type"] == "attention":
            for n, c in (("q", H * D), ("k", m["kv_heads"] * D), ("v", m["kv_heads"] * E)):
                mat(f"{p}.mix.{n}", c, W)
                vec(f"{p}.mix.{n}.b", c, 0.0, 0.5)
            vec(p + ".mix.q.norm", H * D, 1.5, 0.3)
            vec(p + ".mix.k.norm", m["kv_heads"] * D, 1.5, 0.3)
        elif L["type"] == "latent_attention":
            mat(p + ".mix.q", H * (D + m["rot_dim"]), W)
            mat(p + ".mix.dkv", m["kv_rank"] + m["rot_dim"], W)
            vec(p + ".mix.dkv.norm", m["kv_rank"], 1.0, 0.2)
            mat(p + ".mix.uk", H * D, m["kv_rank"])
            mat(p + ".mix.uv", H * E, m["kv_rank"])
        else:
            for n, c in (("q", H * D), ("k", H * D), ("v", H * E), ("g", H * E)):
                mat(f"{p}.mix.{n}", c, W)
        if L["type"] != "retention":
            vec(p + ".mix.sink", H, 0.5, 1.0)
            mat(p + ".mix.g", H, W, std=2.0 / math.sqrt(W))
        mat(p + ".mix.o", W, H * E)
        if f is not None:
            vec(p + ".norm2", W, 1.0, 0.2)
            mat(p + ".mlp.up", f["ff"], W)
            mat(p + ".mlp.down", W, f["ff"])
    vec("final.norm", W, 1.0, 0.2)
    mat("head", V, W)
    return w
