"""Small Sogidra configurations and the plumbing the Sogidra tests share."""
from __future__ import annotations

import math

import pytest
import torch

import sogidra_oracle as S

# (device, dtype): 32-bit on the CPU, 32-bit and bf16 on the GPU
ARMS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
        pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
        pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def pooled(heads, kv_heads, dim, size, pool, cap=30.0, scale=None):
    return "attention_2", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "softcap": float(cap),
                           "mask": {"size": size, "pool": pool}, "scale": scale if scale is not None else 2.0 / math.sqrt(dim)}


def diff(heads, kv_heads, dim, vdim, d, temp=None, kv_from=None, scale=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "diff": d, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}
    if temp is not None:
        m["q_temp"] = {"every": temp[0], "coef": float(temp[1])}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return "attention", m


def config(width, vocab, layers, eps=1e-5, positions=512):
    """``layers``: ``((type, mixer), width of the feed-forward or 0)``."""
    return {"architecture": "Sogidra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "max_positions": positions,
            "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None} for (t, m), ff in layers]}


def cases():
    return {
        # every branch: both mixers, shared keys, with and without a feed-forward, sizes and constants that differ
        "mixed": config(96, 203, [(pooled(6, 2, 20, 11, 5, cap=9.0), 72), (diff(4, 2, 12, 20, 0.35, temp=(7, 0.6)), 56),
                                  (pooled(4, 4, 16, 29, 3, cap=4.0, scale=0.9), 0), (diff(4, 2, 12, 20, 0.45, temp=(16, 0.2), kv_from=1), 88),
                                  (diff(4, 1, 18, 14, 0.1), 40), (diff(8, 2, 12, 20, 0.25, temp=(5, 1.0), kv_from=1), 0),
                                  (pooled(3, 1, 12, 7, 16), 64)], eps=1e-3),
        # a window of one token, blocks of one token, single heads
        "one": config(64, 90, [(pooled(1, 1, 8, 1, 1), 16), (diff(1, 1, 8, 24, 0.5, temp=(1, 0.3)), 24), (pooled(2, 1, 8, 2, 1), 0)]),
        # head sizes of a real model; windows and blocks across tile borders
        "wide": config(128, 160, [(pooled(4, 2, 128, 70, 4, scale=0.15), 192), (diff(4, 2, 64, 128, 0.4, temp=(32, 0.5)), 128),
                                  (pooled(4, 1, 64, 20, 64, scale=0.3), 160), (diff(4, 2, 64, 128, 0.7, kv_from=1), 128)]),
        # what the tensor-core kernels do not take: wide heads, many query heads to a key head
        "broad": config(72, 150, [(pooled(20, 1, 24, 9, 2), 24), (diff(2, 1, 80, 136, 0.3, temp=(4, 0.4)), 40), (pooled(2, 2, 160, 17, 6, scale=0.2), 0),
                                  (diff(20, 1, 16, 24, 0.45), 16)]),
        # nothing is a multiple of 8
        "ragged": config(100, 333, [(diff(10, 5, 9, 22, 0.2, temp=(3, 0.7)), 30), (pooled(3, 3, 14, 17, 7, cap=2.0), 50), (diff(10, 5, 9, 22, 0.8, kv_from=0), 0),
                                    (pooled(5, 1, 18, 40, 13), 70)]),
    }


def model_from(cfg, weights, dtype, device):
    """The product model holding ``weights``, through its own checkpoint names."""
    from jetspec_b200.models import SogidraConfig, SogidraForCausalLM
    from jetspec_b200.models.sogidra import checkpoint_to_parameter as remap
    c = SogidraConfig.from_dict(cfg)
    m = SogidraForCausalLM._empty(c, dtype, device)
    params = m.state_dict()
    assert {remap(k)[0] for k in weights} == set(params) - {"lm_head.weight"}
    with torch.no_grad():
        for k, v in weights.items():
            params[remap(k)[0]].copy_(v.to(dtype))
    return m.eval()


def engine_from(cfg, weights, arm, **kw):
    from jetspec_b200 import JetSpecEngine
    device, dtype = arm
    return JetSpecEngine(model_from(cfg, weights, dtype, device), device=device, dtype=dtype, **kw)


def margin_weights(cfg, seed):
    """Random weights whose greedy choice has a wide margin (bf16 rounding cannot flip it): the sublayers add little to the
    stream, and every position's vector points at a token of its own."""
    w = S.random_weights(cfg, seed=seed)
    for k in w:
        if k.endswith(("norm1b", "norm2b")):
            w[k] = (w[k] * 0.1 - 0.9).to(torch.bfloat16).double()
        elif k.endswith("dwa"):
            w[k][:-1] *= 0.1
    g = torch.Generator().manual_seed(seed)
    w["pos"] = (1.5 * w["embed"][torch.randint(0, cfg["vocab"], (cfg["max_positions"],), generator=g)]).to(torch.bfloat16).double()
    return w


_CACHE: dict = {}


def oracle_logits(key, cfg, weights, tokens):
    """Oracle logits in double precision, computed once per (case, tokens)."""
    k = (key, tuple(tokens))
    if k not in _CACHE:
        _CACHE[k] = S.forward(tokens, weights, cfg)
    return _CACHE[k]


def row_errors(got, want):
    """Per row: rms of the difference over the rms of all expected values (means taken off)."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / scale


def assert_rows(got, want, dtype, what="", bf16=0.04):
    assert got.shape == want.shape
    e = row_errors(got, want)
    assert e.max() < (5e-5 if dtype == torch.float32 else bf16), (what, float(e.max()), int(e.argmax()), len(e))


def prompt(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(900 + seed)).tolist()


def portions(n, sizes):
    """Cut ``n`` into portions of the given sizes, repeated."""
    out, i = [], 0
    while n > 0:
        c = min(n, sizes[i % len(sizes)])
        out.append(c)
        n -= c
        i += 1
    return out


def replay(eng, schedule, requests):
    """Feed ``requests`` (name -> tokens) in portions: ``schedule`` is a list of steps, a step a list of (name, count).
    A request is freed with its last token.  Returns name -> logits of all its tokens."""
    at, sid, out = {n: 0 for n in requests}, {}, {n: [] for n in requests}
    for step in schedule:
        entries = []
        for name, count in step:
            if name not in sid:
                sid[name] = eng._new_seq_id()
            toks = requests[name][at[name]:at[name] + count]
            entries.append((sid[name], toks, list(range(len(toks)))))
        lg, r = eng.step(entries), 0
        for (name, _), (_, toks, _) in zip(step, entries):
            out[name].append(lg[r:r + len(toks)].float().cpu())
            r += len(toks)
            at[name] += len(toks)
            if at[name] == len(requests[name]):
                eng.pool.free(sid[name])
    assert all(at[n] == len(requests[n]) for n in requests)
    return {n: torch.cat(v) for n, v in out.items()}
