"""Small Kizezen configurations and the plumbing the Kizezen tests share."""
from __future__ import annotations

import math

import pytest
import torch

import kizezen_oracle as K

# (device, dtype): 32-bit on the CPU, 32-bit and bf16 on the GPU
ARMS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
        pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
        pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def rot(dims, base, **scaling):
    r = {"dims": dims, "base": float(base)}
    if scaling:
        r["scaling"] = {k: float(v) for k, v in scaling.items()}
    return r


def band(factor, low, high, original):
    return dict(factor=factor, low=low, high=high, original=original)


def ramp(factor, original, fast, slow):
    return dict(factor=factor, original=original, fast=fast, slow=slow)


def window(heads, kv_heads, dim, vdim, size, keep, r, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "rot": r,
                         "mask": {"size": size, "keep_first": keep}, "scale": scale if scale is not None else 1.0 / math.sqrt(dim)}


def latent(heads, dim, vdim, kv_rank, r, scale=None):
    return "latent_attention", {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "rot_dim": r["dims"], "rot": r,
                                "scale": scale if scale is not None else 1.0 / math.sqrt(dim + r["dims"])}


def retention(dim, vdim, decay, r):
    return "retention", {"heads": len(decay), "dim": dim, "vdim": vdim, "decay": [float(x) for x in decay], "rot": r}


def config(width, vocab, layers, eps=1e-5, embed=1.0, logit=1.0):
    """``layers``: ``((type, mixer), width of the feed-forward or 0)``."""
    return {"architecture": "Kizezen", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": embed},
            "logit_scale": logit, "layers": [{"type": t, "mixer": m, "mlp": {"kind": "dense", "ff": ff} if ff else None}
                                             for (t, m), ff in layers]}


def cases():
    return {
        # every branch: all mixers, with and without a feed-forward, sizes and constants that differ from layer to layer
        "mixed": config(96, 203, [(retention(12, 20, [0.5, 0.9, 0.999], rot(8, 1e3)), 72),
                                  (window(6, 2, 20, 28, 11, 3, rot(12, 1e4, **band(8, 1, 4, 64))), 56),
                                  (latent(5, 12, 20, 40, rot(8, 1e3, **ramp(4, 64, 8, 1))), 88),
                                  (window(4, 4, 16, 16, 29, 0, rot(16, 500), scale=0.4), 0),
                                  (retention(20, 12, [1.0, 0.3, 0.75, 0.97], rot(20, 1e4)), 0),
                                  (latent(3, 16, 12, 24, rot(6, 1e4), scale=0.15), 40)], eps=1e-3, embed=0.7, logit=1.7),
        # a window of one token, one head, more kept tokens than the window holds
        "one": config(64, 90, [(window(1, 1, 8, 24, 1, 9, rot(2, 1e4)), 16), (latent(1, 8, 8, 8, rot(2, 1e4, **ramp(2, 32, 4, 1))), 24),
                               (retention(8, 8, [0.8], rot(2, 1e4)), 16)], embed=3.0, logit=0.3),
        # head sizes of a real model
        "wide": config(128, 160, [(window(4, 2, 128, 128, 70, 66, rot(64, 1e6, **band(8, 1, 4, 64))), 192),
                                  (latent(4, 96, 128, 256, rot(32, 1e4, **ramp(16, 32, 16, 1))), 128),
                                  (retention(128, 256, [0.97, 0.995], rot(128, 1e4)), 160),
                                  (latent(8, 64, 64, 512, rot(64, 1e4)), 0)], embed=0.5),
        # what the tensor-core kernels do not take: wide heads, many query heads to a key head, very wide rows
        "broad": config(72, 150, [(window(20, 1, 24, 16, 9, 2, rot(8, 1e4)), 24), (window(2, 1, 160, 136, 40, 5, rot(32, 1e4)), 0),
                                  (latent(2, 136, 144, 700, rot(16, 1e4)), 40), (retention(200, 300, [0.9, 0.99], rot(64, 1e4)), 16)]),
        # nothing is a multiple of 8, no rotated dimension in the third layer
        "ragged": config(100, 333, [(window(10, 5, 18, 22, 17, 5, rot(6, 1e4)), 30), (retention(14, 10, [0.6, 0.93, 0.99], rot(6, 1e3)), 50),
                                    (window(3, 1, 12, 10, 25, 1, rot(0, 1e4)), 0), (latent(3, 10, 14, 36, rot(10, 1e4, **ramp(40, 16, 4, 2))), 70)]),
    }


def model_from(cfg, weights, dtype, device):
    """The product model holding ``weights``, through its own checkpoint names."""
    from jetspec_b200.models import KizezenConfig, KizezenForCausalLM
    from jetspec_b200.models.kizezen import checkpoint_to_parameter
    c = KizezenConfig.from_dict(cfg)
    m, remap = KizezenForCausalLM._empty(c, dtype, device), checkpoint_to_parameter(c)
    params = m.state_dict()
    assert {remap(k)[0] for k in weights} == set(params)
    with torch.no_grad():
        for k, v in weights.items():
            params[remap(k)[0]].copy_(v.to(dtype))
    return m.eval()


def engine_from(cfg, weights, arm, **kw):
    from jetspec_b200 import JetSpecEngine
    device, dtype = arm
    return JetSpecEngine(model_from(cfg, weights, dtype, device), device=device, dtype=dtype, **kw)


def margin_weights(cfg, seed):
    """Random weights whose greedy choice has a wide margin (bf16 rounding cannot flip it): the sublayers add little to
    the stream, and the head scores the successor of the stream's own token."""
    w = K.random_weights(cfg, seed=seed)
    for k in w:
        if k.endswith((".mix.o", ".mlp.down")):
            w[k] = (w[k] * 0.1 * cfg["embedding"]["scale"]).to(torch.bfloat16).double()
    w["head"] = w["embed"].roll(1, 0)
    return w


_CACHE: dict = {}


def oracle_logits(key, cfg, weights, tokens):
    """Oracle logits in double precision, computed once per (case, tokens)."""
    k = (key, tuple(tokens))
    if k not in _CACHE:
        _CACHE[k] = K.forward(tokens, weights, cfg)
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
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(700 + seed)).tolist()


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
