"""Small Zasipel configurations and the plumbing the Zasipel tests share."""
from __future__ import annotations

import math

import pytest
import torch

import zasipel_oracle as Z

# (device, dtype): 32-bit on the CPU, 32-bit and bf16 on the GPU
ARMS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
        pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
        pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def window(heads, kv_heads, dim, vdim, size, rot, base=1e4, scale=None):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": size},
            "rot": {"dims": rot, "base": base}, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}


def delta(heads, kv_heads, dim, vdim, conv):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}


def moe(experts, top, ff, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, eps=1e-5):
    """``layers``: ``(window or None, delta, feed-forward or None)``; without a window the decay is per channel."""
    c = {"architecture": "Zasipel", "width": width, "vocab": vocab, "norm": {"eps": eps}, "layers": []}
    for win, d, f in layers:
        c["layers"].append({"type": "parallel" if win else "channel_delta", "mixer": {"left": win, "right": d} if win else d, "mlp": f})
    return c


def cases():
    return {
        # every branch: both mixers, with and without a feed-forward, sizes that differ from layer to layer
        "mixed": config(96, 203, [(window(6, 2, 20, 28, 11, 12), delta(4, 2, 12, 20, 4), moe(7, 3, 24, 40)),
                                  (None, delta(3, 3, 24, 16, 3), moe(5, 2, 32)),
                                  (window(4, 4, 16, 16, 29, 16, base=500.0, scale=0.4), delta(2, 1, 16, 36, 2), None),
                                  (None, delta(4, 2, 20, 12, 4), None)], eps=1e-3),
        # a window of one token, a convolution of one tap, one head, one expert a token
        "one": config(64, 90, [(window(1, 1, 8, 24, 1, 2), delta(1, 1, 8, 8, 1), moe(3, 1, 16, 24)),
                               (None, delta(1, 1, 16, 40, 1), moe(4, 4, 16))]),
        # head sizes of a real model; long taps
        "wide": config(128, 160, [(window(4, 2, 128, 128, 70, 64, base=1e6), delta(2, 1, 128, 128, 6), moe(4, 2, 64, 64)),
                                  (None, delta(2, 2, 96, 128, 5), moe(4, 2, 72))]),
        # heads wider than the tensor-core kernel takes, many query heads to a key head, more experts than lanes
        "broad": config(72, 150, [(window(20, 1, 24, 16, 9, 8), delta(2, 2, 200, 40, 3), moe(70, 5, 16, 24)),
                                  (window(2, 1, 160, 136, 40, 32), delta(3, 3, 40, 144, 3), None)]),
        # nothing is a multiple of 8, no rotated dimension in the second layer
        "ragged": config(100, 333, [(window(10, 5, 18, 22, 17, 6), delta(5, 5, 10, 14, 4), moe(9, 2, 20, 28)),
                                    (window(3, 1, 12, 10, 25, 0), delta(3, 1, 14, 6, 3), moe(2, 2, 36, 12))]),
    }


def model_from(cfg, weights, dtype, device):
    """The product model holding ``weights``, through its own checkpoint names."""
    from jetspec_b200.models import ZasipelConfig, ZasipelForCausalLM
    from jetspec_b200.models.zasipel import checkpoint_to_parameter
    m = ZasipelForCausalLM._empty(ZasipelConfig.from_dict(cfg, shape_of=lambda n: weights[n].shape), dtype, device)
    params = m.state_dict()
    with torch.no_grad():
        for k, v in weights.items():
            name, index = checkpoint_to_parameter(k)
            dst = params[name] if index is None else params[name][index]
            dst.copy_(v.to(dst.dtype).view(dst.shape))
    return m.eval()


def engine_from(cfg, weights, arm, **kw):
    from jetspec_b200 import JetSpecEngine
    device, dtype = arm
    return JetSpecEngine(model_from(cfg, weights, dtype, device), device=device, dtype=dtype, **kw)


def margin_weights(cfg, seed):
    """Random weights whose greedy choice has a wide margin (bf16 rounding cannot flip it): the sublayers add little to
    the stream, and the head scores the successor of the stream's own token."""
    w = Z.random_weights(cfg, seed=seed)
    for k in w:
        if k.endswith((".norm1", ".norm2")):
            w[k] = (w[k] * 0.15).to(torch.bfloat16).double()
    w["head"] = w["embed"].roll(1, 0)
    return w


_CACHE: dict = {}


def oracle_logits(key, cfg, weights, tokens):
    """Oracle logits in double precision, computed once per (case, tokens)."""
    k = (key, tuple(tokens))
    if k not in _CACHE:
        _CACHE[k] = Z.forward(tokens, weights, cfg)
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
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(300 + seed)).tolist()


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
