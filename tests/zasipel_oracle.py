"""Plain, slow statement of the Zasipel design: one function per mechanism, one sequence at a time, no cache.

Written from the equations alone; it shares no code with ``jetspec_b200``.  Everything runs in the dtype of the weights
handed in (float64 in most tests), so it is the yardstick both for the 32-bit and the bf16 product paths.

Notation: ``x`` is the residual stream ``(T, width)``, ``h`` a sublayer's input, ``w`` a dict of weight tensors with the
checkpoint's names, linear weights ``(out, in)``; row ``t`` of a matrix belongs to token ``t``.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------ pieces
def rms(x, eps):
    """``x`` divided by its root mean square over the last axis."""
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) / x.shape[-1] + eps)


def silu(z):
    return z / (1.0 + torch.exp(-z))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def softplus(z):
    return torch.clamp(z, min=0.0) + torch.log1p(torch.exp(-z.abs()))


def rotate(x, dims, base, positions):
    """Rotate neighbours ``(2i, 2i + 1)`` of the first ``dims`` entries of every head, ``x (T, heads, dim)``."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * float(base) ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


def short_conv(y, taps):
    """``silu`` of a causal convolution per channel: ``taps (channels, n)``, last column on the current row."""
    T, n = y.shape[0], taps.shape[1]
    out = torch.zeros_like(y)
    for t in range(T):
        for j in range(n):
            s = t - (n - 1) + j
            if s >= 0:
                out[t] += taps[:, j] * y[s]
    return silu(out)


def delta_rule(q, k, v, g, beta):
    """The gated delta rule of one head.  ``q, k (T, dim)``, ``v (T, vdim)``, ``g (T, dim)`` decays, ``beta (T,)``.
    Returns the read-outs ``(T, vdim)``."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype)
    out = torch.zeros(q.shape[0], v.shape[1], dtype=q.dtype)
    for t in range(q.shape[0]):
        S = g[t][:, None] * S
        u = beta[t] * (v[t] - S.T @ k[t])
        S = S + torch.outer(k[t], u)
        out[t] = S.T @ q[t]
    return out


# ------------------------------------------------------------------ mixers
def window_attention(h, w, p, m, eps, drop=None):
    """Sliding-window attention with a valueless sink of score 0.  ``drop``: an (i, j) pair made invisible, for tests
    that plant a fault; ``m["no_sink"]`` leaves the sink out likewise."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + ".q"].T + w[p + ".q.b"]).view(T, H, D)
    k = (h @ w[p + ".k"].T + w[p + ".k.b"]).view(T, G, D)
    v = (h @ w[p + ".v"].T + w[p + ".v.b"]).view(T, G, V)
    pos = torch.arange(T)
    q = rms(rotate(q, m["rot"]["dims"], m["rot"]["base"], pos), eps)
    k = rms(rotate(k, m["rot"]["dims"], m["rot"]["base"], pos), eps)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for i in range(T):
        js = [j for j in range(max(0, i - m["mask"]["size"] + 1), i + 1) if (i, j) != drop]
        for n in range(H):
            s = (k[js, n // (H // G)] @ q[i, n]) * m["scale"]
            top = torch.clamp(s.max(), min=0.0) if js else torch.zeros((), dtype=h.dtype)
            e = torch.exp(s - top)
            sink = 0.0 if m.get("no_sink") else torch.exp(-top)
            out[i, n] = (e / (sink + e.sum())) @ v[js, n // (H // G)]
    return out.reshape(T, H * V) @ w[p + ".o"].T + w[p + ".o.b"]


def _delta_inputs(h, w, p, m):
    """Convolved and normalised ``q, k (T, heads, dim)``, ``v (T, heads, vdim)`` and ``beta (T, heads)``."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (short_conv(h @ w[f"{p}.{n}"].T, w[f"{p}.{n}.conv"]) for n in "qkv")
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(q.view(T, G, D)) / math.sqrt(D), unit(k.view(T, G, D))
    share = torch.arange(H) // (H // G)
    return q[:, share], k[:, share], v.view(T, H, V), sigmoid(h @ w[p + ".b"].T)


def _delta_output(o, gate, w, p, eps):
    """Per-head norm, gate and output projection of the read-outs ``o (T, heads, vdim)``."""
    T = o.shape[0]
    return (rms(o, eps) * w[p + ".norm"] * gate.view(o.shape)).reshape(T, -1) @ w[p + ".o"].T


def head_delta(h, w, p, m, eps):
    """Delta rule with one decay per head and a silu gate."""
    q, k, v, beta = _delta_inputs(h, w, p, m)
    g = torch.exp(-torch.exp(w[p + ".A_log"]) * softplus(h @ w[p + ".a"].T + w[p + ".dt_bias"]))
    D = m["dim"]
    o = torch.stack([delta_rule(q[:, n], k[:, n], v[:, n], g[:, n, None].expand(-1, D), beta[:, n]) for n in range(m["heads"])], 1)
    return _delta_output(o, silu(h @ w[p + ".g"].T), w, p, eps)


def channel_delta(h, w, p, m, eps):
    """Delta rule with a decay per head and key channel and a sigmoid gate, both through a low rank."""
    T, H, D = h.shape[0], m["heads"], m["dim"]
    q, k, v, beta = _delta_inputs(h, w, p, m)
    z = (h @ w[p + ".a1"].T) @ w[p + ".a2"].T + w[p + ".dt_bias"]
    g = torch.exp(-torch.exp(w[p + ".A_log"])[:, None] * softplus(z).view(T, H, D))
    o = torch.stack([delta_rule(q[:, n], k[:, n], v[:, n], g[:, n], beta[:, n]) for n in range(H)], 1)
    return _delta_output(o, sigmoid((h @ w[p + ".g1"].T) @ w[p + ".g2"].T), w, p, eps)


def parallel(h, w, p, m, eps, drop=None):
    """Window attention and head-decay delta rule side by side, each normed over the width, averaged."""
    left = window_attention(h, w, p + ".left", m["left"], eps, drop)
    right = head_delta(h, w, p + ".right", m["right"], eps)
    return 0.5 * (rms(left, eps) * w[p + ".left.out"] + rms(right, eps) * w[p + ".right.out"])


# ------------------------------------------------------------------ feed-forward
def expert(h, w, p):
    return (silu(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def table_moe(h, w, p, mlp, tokens):
    """Experts named by a table of token ids, equal weights, plus a shared expert."""
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        for e in w[p + ".table"][tok].long().tolist():
            out[t] += expert(h[t], w, f"{p}.e{e}") / mlp["router"]["top"]
    if mlp.get("shared"):
        out = out + expert(h, w, p + ".shared")
    return out


# ------------------------------------------------------------------ the decoder
def layer(x, w, i, cfg, tokens, drop=None):
    """Both sublayers read the stream itself; each one's output is normed before it is added."""
    L, p, eps = cfg["layers"][i], f"l{i}", cfg["norm"]["eps"]
    if L["type"] == "parallel":
        y = parallel(x, w, p + ".mix", L["mixer"], eps, drop)
    else:
        y = channel_delta(x, w, p + ".mix", L["mixer"], eps)
    x = x + rms(y, eps) * w[p + ".norm1"]
    if L["mlp"] is not None:
        x = x + rms(table_moe(x, w, p + ".mlp", L["mlp"], tokens), eps) * w[p + ".norm2"]
    return x


def forward(tokens, w, cfg, streams=None, drop=None):
    """Logits ``(T, vocab)`` of one whole sequence; ``streams`` collects the residual stream after every layer."""
    tokens = [int(t) for t in tokens]
    x = w["embed"][tokens]
    for i in range(len(cfg["layers"])):
        x = layer(x, w, i, cfg, tokens, drop)
        if streams is not None:
            streams.append(x)
    return (rms(x, cfg["norm"]["eps"]) * w["final.norm"]) @ w["head"].T


def greedy(tokens, w, cfg, n):
    """``n`` greedy continuations, recomputing the whole sequence for every token."""
    ids = list(tokens)
    for _ in range(n):
        ids.append(int(forward(ids, w, cfg)[-1].argmax()))
    return ids[len(tokens):]


# ------------------------------------------------------------------ random models for the tests
def random_weights(cfg, ranks=(5, 7), seed=0, dtype=torch.float64):
    """Weights of every tensor ``cfg`` implies, rounded to bf16 (what a checkpoint holds).  ``ranks``: the low ranks of
    the decay and of the gate of channel-decay layers.  Decays spread from forgetting within a token to remembering
    hundreds."""
    g = torch.Generator().manual_seed(seed)
    w, W, V = {}, cfg["width"], cfg["vocab"]
    bf = lambda x: x.to(torch.bfloat16).to(dtype)

    def mat(name, *shape, std=None):
        w[name] = bf(torch.randn(*shape, generator=g) * (std if std is not None else 1.0 / math.sqrt(shape[-1])))

    def vec(name, n, around, spread):
        w[name] = bf(around + spread * torch.randn(n, generator=g))

    def delta(p, m, channel):
        kd, vd = m["kv_heads"] * m["dim"], m["heads"] * m["vdim"]
        for n, c in (("q", kd), ("k", kd), ("v", vd)):
            mat(f"{p}.{n}", c, W)
            mat(f"{p}.{n}.conv", c, m["conv"], std=0.6)
        mat(p + ".b", m["heads"], W)
        w[p + ".A_log"] = bf(torch.linspace(-5.0, 1.5, m["heads"]))
        vec(p + ".norm", m["vdim"], 1.0, 0.2)
        if channel:
            mat(p + ".a1", ranks[0], W)
            mat(p + ".a2", m["heads"] * m["dim"], ranks[0])
            vec(p + ".dt_bias", m["heads"] * m["dim"], -1.0, 1.5)
            mat(p + ".g1", ranks[1], W)
            mat(p + ".g2", vd, ranks[1])
        else:
            mat(p + ".a", m["heads"], W)
            vec(p + ".dt_bias", m["heads"], -1.0, 1.0)
            mat(p + ".g", vd, W)
        mat(p + ".o", W, vd)

    def experts(p, f):
        for n, c in (("gate", f), ("up", f)):
            mat(f"{p}.{n}", c, W)
        mat(p + ".down", W, f)

    mat("embed", V, W, std=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", L["mixer"], L["mlp"]
        vec(p + ".norm1", W, 1.0, 0.2)
        if L["type"] == "parallel":
            a = m["left"]
            for n, c, k in (("q", a["heads"] * a["dim"], W), ("k", a["kv_heads"] * a["dim"], W), ("v", a["kv_heads"] * a["vdim"], W),
                            ("o", W, a["heads"] * a["vdim"])):
                mat(f"{p}.mix.left.{n}", c, k)
                vec(f"{p}.mix.left.{n}.b", c, 0.0, 0.5)
            delta(p + ".mix.right", m["right"], False)
            vec(p + ".mix.left.out", W, 1.0, 0.2)
            vec(p + ".mix.right.out", W, 1.0, 0.2)
        else:
            delta(p + ".mix", m, True)
        if f is None:
            continue
        vec(p + ".norm2", W, 1.0, 0.2)
        for e in range(f["router"]["experts"]):
            experts(f"{p}.mlp.e{e}", f["expert"]["ff"])
        order = torch.rand(V, f["router"]["experts"], generator=g).argsort(-1)
        w[p + ".mlp.table"] = order[:, : f["router"]["top"]].to(torch.int32)
        if f.get("shared"):
            experts(p + ".mlp.shared", f["shared"]["ff"])
    vec("final.norm", W, 1.0, 0.2)
    mat("head", V, W)
    return w
