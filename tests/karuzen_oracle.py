"""Plain, slow statement of the Karuzen design: one function per mechanism, one sequence at a time, no cache.

Written from the equations alone; it shares no code with ``jetspec_b200``.  Everything runs in the dtype of the
weights handed in (float64 in most tests), so it is the yardstick both for the 32-bit and the bf16 product paths.

Notation: ``x`` is the residual stream ``(T, width)``, ``h`` a sublayer input, ``w`` a dict of weight tensors with the
checkpoint's names, linear weights ``(out, in)``.
"""
from __future__ import annotations

import math

import torch


def dynamic_tanh(x, alpha, weight, bias):
    """``tanh(alpha x) * weight + bias``, elementwise; ``alpha`` is one number."""
    return torch.tanh(alpha * x) * weight + bias


def rms_norm(x, weight, eps):
    ms = (x * x).sum(-1, keepdim=True) / x.shape[-1]
    return x / torch.sqrt(ms + eps) * weight


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def squared_relu(z):
    return torch.clamp(z, min=0.0) ** 2


def latent_attention(h, w, p, mixer, eps, visible=None):
    """Attention through two latents.  ``visible`` ``(T, T)`` bool replaces the causal mask when given."""
    T, H, D, V = h.shape[0], mixer["heads"], mixer["dim"], mixer["vdim"]
    cq = rms_norm(h @ w[p + ".dq"].T, w[p + ".dq.norm"], eps)
    c = rms_norm(h @ w[p + ".dkv"].T, w[p + ".dkv.norm"], eps)
    q = (cq @ w[p + ".uq"].T).view(T, H, D)
    k = (c @ w[p + ".uk"].T).view(T, H, D)
    v = (c @ w[p + ".uv"].T).view(T, H, V)
    out = torch.zeros(T, H, V, dtype=h.dtype)
    for i in range(T):
        js = range(i + 1) if visible is None else [j for j in range(T) if bool(visible[i, j])]
        js = torch.tensor(list(js))
        for n in range(H):
            s = (k[js, n] @ q[i, n]) * mixer["scale"]
            e = torch.exp(s - s.max())
            out[i, n] = (e / e.sum()) @ v[js, n]
    return out.reshape(T, H * V) @ w[p + ".o"].T


def dense_mlp(h, w, p):
    return (gelu_tanh(h @ w[p + ".gate"].T) * (h @ w[p + ".up"].T)) @ w[p + ".down"].T


def expert(h, w, p):
    return squared_relu(h @ w[p + ".up"].T) @ w[p + ".down"].T


def route(h_row, w, p, router):
    """``[(expert, weight), ...]`` of one token, largest choice score first."""
    s = torch.sigmoid(w[p + ".router"] @ h_row)
    choice = s + w[p + ".correction"]
    chosen = sorted(range(router["experts"]), key=lambda e: (-float(choice[e]), e))[: router["top"]]
    total = sum(float(s[e]) for e in chosen) + 1e-20
    return [(e, float(s[e]) / total * router["scale"]) for e in chosen]


def moe_mlp(h, w, p, mlp):
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, g in route(h[t], w, p, mlp["router"]):
            out[t] += g * expert(h[t], w, f"{p}.e{e}")
        if mlp.get("shared"):
            out[t] += torch.sigmoid(w[p + ".shared.sg"] @ h[t]) * expert(h[t], w, p + ".shared")
    return out


def layer(x, w, i, cfg, visible=None):
    """``x + mixer(h) + ff(h)`` with ``h`` the block's single normalised input."""
    L, p = cfg["layers"][i], f"l{i}"
    h = dynamic_tanh(x, w[p + ".norm1.alpha"], w[p + ".norm1"], w[p + ".norm1.b"])
    y = latent_attention(h, w, p + ".mix", L["mixer"], cfg["norm"]["eps"], visible)
    if L["mlp"] is not None:
        y = y + (dense_mlp(h, w, p + ".mlp") if L["mlp"]["kind"] == "dense" else moe_mlp(h, w, p + ".mlp", L["mlp"]))
    return x + y


def schedule(cfg):
    """``[(layer, add the embedding output first?), ...]`` in the order the layers run."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    runs = [(i, False) for i in range(loop["start"])]
    for r in range(loop["times"]):
        runs += [(i, r > 0 and i == loop["start"]) for i in range(loop["start"], loop["stop"])]
    return runs + [(i, False) for i in range(loop["stop"], n)]


def forward(tokens, w, cfg, visible=None, streams=None):
    """Logits ``(T, vocab)`` of one whole sequence; ``streams`` collects the residual stream after every layer run."""
    e = w["embed"][torch.as_tensor(tokens)]
    x = e.clone()
    for i, again in schedule(cfg):
        if again:
            x = x + e
        x = layer(x, w, i, cfg, visible)
        if streams is not None:
            streams.append(x)
    return dynamic_tanh(x, w["final.norm.alpha"], w["final.norm"], w["final.norm.b"]) @ w["embed"].T


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
    w, W = {}, cfg["width"]

    def mat(name, *shape, std=None):
        std = std if std is not None else 1.0 / math.sqrt(shape[-1])
        w[name] = (torch.randn(*shape, generator=g) * std).to(torch.bfloat16).to(dtype)

    def vec(name, n, around, spread):
        w[name] = (around + spread * torch.randn(n, generator=g)).to(torch.bfloat16).to(dtype)

    def dyt(name):
        vec(name, W, 1.0, 0.2)
        vec(name + ".b", W, 0.0, 0.2)
        w[name + ".alpha"] = torch.tensor(0.4 + 0.5 * torch.rand(1, generator=g).item()).to(torch.bfloat16).to(dtype)

    mat("embed", cfg["vocab"], W, std=1.0)
    for i, L in enumerate(cfg["layers"]):
        p, m, f = f"l{i}", L["mixer"], L["mlp"]
        dyt(p + ".norm1")
        mat(p + ".mix.dq", m["q_rank"], W)
        vec(p + ".mix.dq.norm", m["q_rank"], 1.0, 0.2)
        mat(p + ".mix.uq", m["heads"] * m["dim"], m["q_rank"])
        mat(p + ".mix.dkv", m["kv_rank"], W)
        vec(p + ".mix.dkv.norm", m["kv_rank"], 1.0, 0.2)
        mat(p + ".mix.uk", m["heads"] * m["dim"], m["kv_rank"])
        mat(p + ".mix.uv", m["heads"] * m["vdim"], m["kv_rank"])
        mat(p + ".mix.o", W, m["heads"] * m["vdim"])
        if f is None:
            continue
        if f["kind"] == "dense":
            mat(p + ".mlp.gate", f["ff"], W)
            mat(p + ".mlp.up", f["ff"], W)
            mat(p + ".mlp.down", W, f["ff"])
            continue
        for e in range(f["router"]["experts"]):
            mat(f"{p}.mlp.e{e}.up", f["expert"]["ff"], W)
            mat(f"{p}.mlp.e{e}.down", W, f["expert"]["ff"])
        mat(p + ".mlp.router", f["router"]["experts"], W)
        vec(p + ".mlp.correction", f["router"]["experts"], 0.0, 0.3)
        if f.get("shared"):
            mat(p + ".mlp.shared.up", f["shared"]["ff"], W)
            mat(p + ".mlp.shared.down", W, f["shared"]["ff"])
            mat(p + ".mlp.shared.sg", 1, W)
    dyt("final.norm")
    return w
