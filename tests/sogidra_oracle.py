"""Plain, slow statement of the Sogidra design: one function per mechanism, one sequence at a time, no cache.

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


def norm(x, w, eps):
    """RMS norm whose weight is stored as its distance from one."""
    return rms(x, eps) * (w + 1.0)


def softplus(z):
    return torch.log1p(torch.exp(z))


def xielu(z, act):
    """Quadratic for positive ``z``, an integrated ELU below; slope 1/2 at zero from both sides."""
    up, down = softplus(act[0]), 0.5 + softplus(act[1])
    return z / 2.0 + torch.where(z > 0, up * z * z, down * (torch.expm1(z.clamp(max=0.0)) - z))


def capped(s, cap):
    return cap * torch.tanh(s / cap)


def temperature(positions, every, coef):
    """Factor on the query at each position: grows with the logarithm of how many times ``every`` fits."""
    return torch.tensor([1.0 + coef * math.log((int(p) + 1) // every + 1) for p in positions], dtype=torch.float64)


def softmax(s):
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


# ------------------------------------------------------------------ differential attention
def differential_keys(h, w, p, m):
    """``(T, G, 2, D)`` keys of the two maps and ``(T, G, V)`` values of a layer that has projections of its own."""
    T, G = h.shape[0], m["kv_heads"]
    return ((h @ w[p + ".k"].T + w[p + ".k.b"]).view(T, G, 2, m["dim"]), (h @ w[p + ".v"].T + w[p + ".v.b"]).view(T, G, m["vdim"]))


def differential_lambda(w, p, m):
    return torch.exp((w[p + ".lq1"] * w[p + ".lk1"]).sum()) - torch.exp((w[p + ".lq2"] * w[p + ".lk2"]).sum()) + m["diff"]


def attention(h, w, p, m, eps, kv=None, fault=None):
    """Causal differential attention without rotation; ``kv``: keys and values of the layer it shares them with.  ``fault``
    (tests that plant one): ``"no_temp"``, ``"no_second_map"``, ``"plain_lambda"`` or a pair ``(i, j)`` whose visibility is
    flipped."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    k, v = differential_keys(h, w, p, m) if kv is None else kv
    q = (h @ w[p + ".q"].T + w[p + ".q.b"]).view(T, H, 2, D)
    if m.get("q_temp") and fault != "no_temp":
        q = q * temperature(range(T), m["q_temp"]["every"], m["q_temp"]["coef"]).to(h.dtype)[:, None, None, None]
    seen = torch.tril(torch.ones(T, T, dtype=torch.bool))
    if isinstance(fault, tuple):
        seen[fault] = ~seen[fault]
    lam = {"no_second_map": 0.0, "plain_lambda": m["diff"]}.get(fault) if isinstance(fault, str) else None
    lam = differential_lambda(w, p, m) if lam is None else lam
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for n in range(H):
        g = n // (H // G)
        a = [softmax((q[:, n, i] @ k[:, g, i].T * m["scale"]).masked_fill(~seen, -math.inf)) @ v[:, g] for i in (0, 1)]
        out[:, n] = rms(a[0] - lam * a[1], eps) * (1.0 - m["diff"])
    return out.reshape(T, H * V) @ w[p + ".o"].T


# ------------------------------------------------------------------ window attention with pooled blocks
def window_and_blocks(T, size, P):
    """Visibility of the ``T`` tokens and of the ``T // P`` whole blocks for every row."""
    i, j, b = torch.arange(T)[:, None], torch.arange(T)[None], torch.arange(T // P)[None]
    return (j <= i) & (i - j < size), (b + 1) * P - 1 <= i - size


def pooled_attention(h, w, p, m, eps, fault=None):
    """Attention over the last tokens and the means of whole blocks behind them, in one softmax with capped scores; values are
    the keys ahead of their norm.  ``fault``: ``"no_cap"``, ``"no_blocks"``, ``"normed_values"``, or ``("key" | "block", i, j)``
    whose visibility is flipped."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = rms((h @ w[p + ".q"].T).view(T, H, D), eps)
    v = (h @ w[p + ".k"].T).view(T, G, D)
    k = rms(v, eps)
    if fault == "normed_values":
        v = k
    size, P = m["mask"]["size"], m["mask"]["pool"]
    near, far = window_and_blocks(T, size, P)
    if isinstance(fault, tuple):
        seen = near if fault[0] == "key" else far
        seen[fault[1:]] = ~seen[fault[1:]]
    if fault == "no_blocks":
        far = torch.zeros_like(far)
    n = T // P
    out = torch.zeros(T, H, D, dtype=h.dtype)
    for u in range(H):
        g = u // (H // G)
        kb, vb = (x[: n * P, g].reshape(n, P, D).mean(1) for x in (k, v))
        s = torch.cat((q[:, u] @ k[:, g].T, q[:, u] @ kb.T), -1) * m["scale"]
        if fault != "no_cap":
            s = capped(s, m["softcap"])
        a = softmax(s.masked_fill(~torch.cat((near, far), -1), -math.inf))
        out[:, u] = a[:, :T] @ v[:, g] + a[:, T:] @ vb
    return out.reshape(T, H * D) @ w[p + ".o"].T


MIXERS = {"attention": attention, "attention_2": pooled_attention}


# ------------------------------------------------------------------ the decoder
def feed_forward(h, w, p):
    return xielu(h @ w[p + ".up"].T, w[p + ".act"]) @ w[p + ".down"].T


def depth_average(history, d):
    """Weighted sum of the embedding output and every layer's result so far."""
    return sum(d[j] * x for j, x in enumerate(history))


def forward(tokens, w, cfg, streams=None, faults=None):
    """Logits ``(T, vocab)`` of one whole sequence; ``streams`` collects what every layer passes on; ``faults`` maps a layer to
    a planted fault of its mixer (or to ``"no_average"``, ``"no_out_norm"``)."""
    eps, T = cfg["norm"]["eps"], len(tokens)
    x = w["embed"][[int(t) for t in tokens]] + w["pos"][:T]
    history, shared = [x], {}
    for i, L in enumerate(cfg["layers"]):
        p, m, fault = f"l{i}", L["mixer"], (faults or {}).get(i)
        mine = fault if fault not in ("no_average", "no_out_norm") else None
        h, more = norm(x, w[p + ".norm1"], eps), {}
        if L["type"] == "attention":
            if m.get("kv_from") is None:
                shared[i] = differential_keys(h, w, p + ".mix", m)
            more["kv"] = shared[i if m.get("kv_from") is None else m["kv_from"]]
        y = MIXERS[L["type"]](h, w, p + ".mix", m, eps, fault=mine, **more)
        x = x + (y if fault == "no_out_norm" else norm(y, w[p + ".norm1b"], eps))
        if L["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, w[p + ".norm2"], eps), w, p + ".mlp"), w[p + ".norm2b"], eps)
        history.append(x)
        if fault != "no_average":
            x = depth_average(history, w[p + ".dwa"])
        if streams is not None:
            streams.append(x)
    return norm(x, w["final.norm"], eps) @ w["embed"].T


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
    mat("pos", cfg["max_positions"], W, std=0.5)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", L["mixer"], L["mlp"]
        H, G, D, E = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
        for n in ("norm1", "norm1b") + (("norm2", "norm2b") if f is not None else ()):
            vec(f"{p}.{n}", W, -0.3 if n.endswith("b") else 0.0, 0.2)
        if L["type"] == "attention":
            for n, c in (("q", 2 * H * D), ("k", 2 * G * D), ("v", G * E)):
                if n == "q" or m.get("kv_from") is None:
                    mat(f"{p}.mix.{n}", c, W)
                    vec(f"{p}.mix.{n}.b", c, 0.0, 0.5)
            for n in ("lq1", "lk1", "lq2", "lk2"):
                vec(f"{p}.mix.{n}", D, 0.3 if n == "lq1" else 0.0, 0.8 / math.sqrt(D) ** 0.5)
        else:
            mat(p + ".mix.q", H * D, W)
            mat(p + ".mix.k", G * D, W)
        mat(p + ".mix.o", W, H * E)
        if f is not None:
            mat(p + ".mlp.up", f["ff"], W)
            mat(p + ".mlp.down", W, f["ff"])
            vec(p + ".mlp.act", 2, 0.5, 0.5)
        d = torch.randn(i + 2, generator=g) * 0.2
        d[-1] += 1.0
        w[p + ".dwa"] = bf(d)
    vec("final.norm", W, 0.0, 0.2)
    return w
