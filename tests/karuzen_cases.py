"""Small Karuzen configurations and the plumbing the Karuzen tests share."""
from __future__ import annotations

import math

import pytest
import torch

import karuzen_oracle as K

# (device, dtype): 32-bit on the CPU, 32-bit and bf16 on the GPU
ARMS = [pytest.param(("cpu", torch.float32), id="cpu-f32"),
        pytest.param(("cuda", torch.float32), id="gpu-f32", marks=pytest.mark.gpu),
        pytest.param(("cuda", torch.bfloat16), id="gpu-bf16", marks=pytest.mark.gpu)]


def mixer(heads, dim, vdim, q_rank, kv_rank, scale=None):
    return {"heads": heads, "dim": dim, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank,
            "scale": scale if scale is not None else 1.5 / math.sqrt(dim)}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, scale, shared=None):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top, "scale": scale}}
    if shared:
        m["shared"] = {"ff": shared}
    return m


def config(width, vocab, layers, loop=None, eps=1e-5):
    c = {"architecture": "Karuzen", "width": width, "vocab": vocab, "norm": {"eps": eps},
         "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}
    if loop:
        c["loop"] = dict(zip(("start", "stop", "times"), loop))
    return c


def cases():
    a, b = mixer(3, 20, 12, 28, 36), mixer(2, 24, 40, 16, 52, scale=0.9)
    wide = mixer(4, 72, 100, 60, 300)
    return {
        # dense, routed, bare layers; a loop in the middle; sizes differ from layer to layer
        "mixed": config(96, 203, [(a, dense(80)), (b, moe(7, 3, 24, 1.4, shared=56)), (a, None), (b, dense(40))], loop=(1, 3, 2), eps=1e-3),
        # every layer routed, no shared expert, one expert a token, the loop reaches from the first to the last layer
        "routed": config(64, 160, [(a, moe(5, 1, 32, 1.0)), (b, moe(4, 4, 16, 0.7))], loop=(0, 2, 3)),
        # no loop, one head, values wider than keys, a latent of three lines
        "plain": config(80, 96, [(mixer(1, 16, 48, 40, 130), dense(64)), (mixer(1, 16, 48, 40, 130), dense(64))]),
        # a loop that runs once; nothing is a multiple of 8
        "ragged": config(100, 333, [(mixer(5, 18, 22, 30, 50), dense(36)), (mixer(5, 18, 22, 30, 50), moe(9, 2, 20, 2.0, shared=28))],
                         loop=(0, 1, 1)),
        # a latent wider than the tensor-core attention takes, more experts than a warp has lanes
        "broad": config(64, 120, [(mixer(2, 12, 12, 20, 520), moe(70, 6, 16, 1.1, shared=16)), (mixer(3, 8, 16, 24, 24), dense(48))]),
        # heads wide enough for the expanded form of long portions, a latent of five lines (two column groups)
        "wide": config(128, 200, [(wide, moe(6, 2, 64, 1.2, shared=64)), (wide, dense(96))], loop=(0, 1, 2)),
    }


def model_from(cfg, weights, dtype, device):
    """The product model holding ``weights``, through its own checkpoint names."""
    from jetspec_b200.models import KaruzenConfig, KaruzenForCausalLM
    from jetspec_b200.models.karuzen import checkpoint_to_parameter
    m = KaruzenForCausalLM._empty(KaruzenConfig.from_dict(cfg), dtype, device)
    params = dict(m.named_parameters())
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


def prompt(n, vocab, seed=0):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist()


def row_errors(got, want):
    """Per row: rms of the difference over the rms of all expected values (means taken off)."""
    got, want = got.double().cpu(), want.double()
    d = got - want
    d = d - d.mean(-1, keepdim=True)
    scale = (want - want.mean(-1, keepdim=True)).pow(2).mean().sqrt()
    return d.pow(2).mean(-1).sqrt() / scale


def assert_rows(got, want, dtype, what=""):
    """32-bit: every row to 5e-5.  bf16: rounding may flip a close routing call, which moves that row (and, less, rows
    that attend to it); nine rows in ten must agree to 4 %, all to 40 %."""
    assert got.shape == want.shape
    e = row_errors(got, want)
    if dtype == torch.float32:
        assert e.max() < 5e-5, (what, e.max(), int(e.argmax()))
    else:
        assert e.quantile(0.9) < 0.04 and e.max() < 0.4, (what, e.quantile(0.9), e.max(), int(e.argmax()))


def replay(eng, schedule, requests, dtype=None):
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
        lg = eng.step(entries)
        r = 0
        for (name, count), (_, toks, _) in zip(step, entries):
            out[name].append(lg[r:r + len(toks)].float().cpu())
            r += len(toks)
            at[name] += len(toks)
            if at[name] == len(requests[name]):
                eng.pool.free(sid[name])
    assert all(at[n] == len(requests[n]) for n in requests)
    return {n: torch.cat(v) for n, v in out.items()}


def portions(n, sizes):
    """Cut ``n`` into portions of the given sizes, repeated."""
    out, i = [], 0
    while n > 0:
        c = min(n, sizes[i % len(sizes)])
        out.append(c)
        n -= c
        i += 1
    return out


_CACHE: dict = {}


def oracle_logits(key, cfg, weights, tokens):
    """Oracle logits in double precision, computed once per (case, tokens)."""
    k = (key, tuple(tokens))
    if k not in _CACHE:
        _CACHE[k] = K.forward(tokens, weights, cfg)
    return _CACHE[k]
