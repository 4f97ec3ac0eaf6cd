"""Prefill and decode throughput of Karuzen beside Qwen3 of equal size, and the roofline of every kernel of a layer.

    python bench.py --design karuzen                 # what this module's main() runs
    python bench.py --design karuzen --part kernels  # per-kernel timings only

Models: random weights, the same width, feed-forward, depth, vocabulary and (for the routed pair) experts in both
families.  ``prefill``: one prompt through the engine's prompt path; ``decode``: replays of the batched one-token graph
the engine's ``generate_batch`` uses, ``batch`` requests at ``context`` cached tokens.  Device time with CUDA events after
warm-up; a step streams the weights of all layers, which are larger than L2.

``kernels``: each kernel captured alone into a graph over enough weight copies to miss L2, its time per launch, and the
roofline time from the bytes and FLOPs the algorithm needs at the measured copy bandwidth and bf16 GEMM rate.
"""
from __future__ import annotations

import json
import os
import sys

import torch

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def peaks():
    """(bytes/s, FLOP/s, where from): the measured copy bandwidth and cuBLAS bf16 burst rate."""
    try:
        d = json.load(open(os.path.join(ROOT, "MEASURED_PEAKS.json")))
        return d["hbm_gbs"] * 1e9, d["bf16_tflops"] * 1e12, "of measured"
    except Exception:
        return 6.65e12, 1.59e15, "of fallback"


def pairs(depth: int):
    """name -> (Karuzen config, Qwen3 config) of equal size."""
    from jetspec_b200.models import KaruzenConfig, KaruzenLayerConfig, LatentAttentionConfig, Qwen3Config, RoutedExpertsConfig

    def kz(width, heads, q_rank, kv_rank, vocab, ff=0, moe=None, loop=None, n=depth):
        mix = LatentAttentionConfig(heads, 128, 128, q_rank, kv_rank, 128 ** -0.5)
        c = KaruzenConfig(vocab_size=vocab, hidden_size=width, layers=[KaruzenLayerConfig(mix, ff, moe) for _ in range(n)])
        if loop:
            c.loop_start, c.loop_stop, c.loop_times = loop
        return c

    def qw(width, heads, kv, vocab, ff, **kw):
        return Qwen3Config(vocab_size=vocab, hidden_size=width, intermediate_size=ff, num_hidden_layers=depth,
                           num_attention_heads=heads, num_key_value_heads=kv, head_dim=128, **kw)

    moe_kw = dict(num_experts=128, num_experts_per_tok=8, moe_intermediate_size=768, model_type="qwen3_moe")
    return {
        "dense 4096": (kz(4096, 32, 1536, 512, 32768, ff=12288), qw(4096, 32, 8, 32768, 12288)),
        "dense 2048": (kz(2048, 16, 768, 512, 32768, ff=6144), qw(2048, 16, 8, 32768, 6144)),
        "routed 2048": (kz(2048, 32, 768, 512, 32768, moe=RoutedExpertsConfig(128, 8, 2.5, 768, 768)), qw(2048, 32, 4, 32768, 6144, **moe_kw)),
        "dense 4096, half the layers run twice": (kz(4096, 32, 1536, 512, 32768, ff=12288, loop=(0, depth // 2, 2), n=depth // 2),
                                                  qw(4096, 32, 8, 32768, 12288)),
    }


def timed(fn, reps=5, warm=3):
    for _ in range(warm):
        fn()
    e = [torch.cuda.Event(enable_timing=True) for _ in range(2)]
    torch.cuda.synchronize()
    e[0].record()
    for _ in range(reps):
        fn()
    e[1].record()
    torch.cuda.synchronize()
    return e[0].elapsed_time(e[1]) / reps


def throughput(name, cfg, prompt=2048, context=2048, batches=(1, 16)):
    from jetspec_b200 import JetSpecEngine
    from jetspec_b200.engine.engine import _OneNode
    from jetspec_b200.engine.fast_round import FastRound
    from jetspec_b200.models import family_of
    model = family_of({"model_type": cfg.model_type}).model_cls.random_init(cfg, seed=0, dtype=torch.bfloat16, device="cuda")
    eng = JetSpecEngine(model, device="cuda", dtype=torch.bfloat16, max_seq_len=max(prompt, context) + 64, max_seqs=max(batches))
    out = {"model": name, "family": cfg.model_type, "layer_runs": cfg.num_hidden_layers, "cache_bytes_per_token": 0}
    eng._ensure_pool((max(prompt, context) + 48) * max(batches), seqs=max(batches))
    pool, fast = eng.pool, FastRound.get(eng)
    held = {id(kv): kv for kv in (*(pool.kv_layers or []), *(pool.kv_blocks or [])) if kv is not None}        # shared pools once
    bufs = [b for b in pool.latent_pools or [] if b is not None] + [b for kv in held.values() for b in kv]
    bufs = bufs or [pool.k_pool, pool.v_pool]
    if pool.states is not None:
        out["state_bytes_per_sequence"] = sum(t[0].numel() * t.element_size() for t in (*pool.states.state, *pool.states.conv) if t is not None)
    out["cache_bytes_per_token"] = sum(b.numel() * b.element_size() for b in bufs) // pool.num_slots
    ids = torch.randint(0, cfg.vocab_size, (1, prompt), generator=torch.Generator().manual_seed(0)).cuda()

    def prefill():
        sid = eng._new_seq_id()
        fast._prefill_kernels(sid, ids, None, prompt)
        pool.free(sid)
    with torch.inference_mode():
        ms = timed(prefill, reps=4)
        out[f"prefill_{prompt}"] = {"ms": round(ms, 3), "tokens_per_s": round(prompt / ms * 1e3)}
        for b in batches:
            sids = [eng._new_seq_id() for _ in range(b)]
            for s in sids:
                pool.reserve(s, context + 16)
                pool.state(s).length = context
            nodes = [_OneNode(1 + i) for i in range(b)]
            fast.batch_verify(sids, nodes, [context] * b, 1)
            g = fast.graphs[("batch", b, 1, (), id(pool))]["graph"]
            ms = timed(g.replay, reps=10)
            out[f"decode_b{b}_ctx{context}"] = {"ms": round(ms, 4), "tokens_per_s": round(b / ms * 1e3, 1)}
            for s in sids:
                pool.free(s)
    from jetspec_b200.ops import cuda_ext
    cuda_ext.check_status("cuda")
    del eng, model, fast
    torch.cuda.empty_cache()
    return out


# ------------------------------------------------------------------ one kernel at a time
def graph_time_us(fns, inner):
    """Time per call of ``fns[i]()`` (one per weight copy), ``inner`` calls round robin inside one graph."""
    for f in fns:
        f()
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for i in range(inner):
            fns[i % len(fns)]()
    return timed(g.replay, reps=5) * 1e3 / inner


def kernel_table(T, context, n_seq):
    """Per-launch times of a layer's kernels for ``T`` rows (``n_seq`` sequences with ``context`` cached tokens each),
    Karuzen at width 4096 / Qwen3-8B sizes, and their rooflines."""
    from jetspec_b200.ops import cuda_ext as X
    bw, fl, note = peaks()
    W, H, R, QR, FF, D = 4096, 32, 512, 1536, 12288, 128
    dev = "cuda"
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(torch.bfloat16)
    rows = []

    def add(name, fns, nbytes, flops, inner=None, like=None):
        us = graph_time_us(fns, inner or 2 * len(fns))
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 4), "like": like})

    def weights(n, k):
        copies = max(2, int(400e6 / (n * k * 2)) + 1)
        return [bf(n, k) for _ in range(min(copies, 24))]

    def gemm_case(name, n, k, call, out_bytes, like=None):
        ws = weights(n, k)
        add(name, [lambda w=w: call(w) for w in ws], (n * k + T * k) * 2 + T * out_bytes, 2 * T * n * k, like=like)

    h, cq = bf(T, W), bf(T, QR)
    n_raw = QR + R
    raw, cat = torch.empty(T, n_raw, device=dev), bf(T, H * D + FF)
    # ---- Qwen3-8B's kernels
    gemm_case("qwen3 qkv GEMM", 6144, W, lambda w: X.gemm(h, w), 6144 * 2)
    xr = bf(T, W)
    att, act = bf(T, W), bf(T, FF)
    gemm_case("qwen3 o GEMM + residual", W, W, lambda w: X.gemm(att, w, out=xr, residual=xr), W * 4)
    if T >= 1024:
        gemm_case("qwen3 gate/up GEMM + SwiGLU", 2 * FF, W, lambda w: X.gemm(h, w, epi=X.EPI_SWIGLU, bn=256, split=1, deep=0), FF * 2)
    else:
        gemm_case("qwen3 gate/up GEMM + SwiGLU", 2 * FF, W, lambda w: X.gemm(h, w, epi=X.EPI_SWIGLU), FF * 2)
    gemm_case("qwen3 down GEMM + residual", W, FF, lambda w: X.gemm(act, w, out=xr, residual=xr), W * 4)
    nw = bf(W)
    add("qwen3 RMSNorm", [lambda: X.rmsnorm(h, nw, 1e-6)], T * W * 4, 0, 8)
    qkv, pos = bf(T, 6144), torch.arange(T, dtype=torch.int32, device=dev)
    S = n_seq * (context + T) + 64
    kp, vp = bf(8, S, D), bf(8, S, D)
    q = bf(T, H, D)
    freq = X.inv_freq(D, 1e6, dev)
    add("qwen3 head norms + RoPE + KV scatter", [lambda: X.qkv_post(qkv, nw[:D], nw[:D], pos, pos, freq, q, kp, vp, H, 8, 1e-6)], T * 6144 * 4, 0, 8)
    per = T // n_seq
    smap = torch.randperm(S, device=dev).to(torch.int32)[: n_seq * (context + per)].view(n_seq, context + per).contiguous()
    srow = torch.arange(n_seq, dtype=torch.int32, device=dev)
    cu = (torch.arange(n_seq + 1, dtype=torch.int32, device=dev) * per).contiguous()
    past = torch.full((n_seq,), context, dtype=torch.int32, device=dev)
    keys = n_seq * per * context + n_seq * per * (per + 1) // 2          # visible (query, key) pairs
    tot = n_seq * (context + per)
    nk = max(1, int(300e6 / (tot * 4096)) + 1)
    pools = [(bf(8, S, D), bf(8, S, D)) for _ in range(min(nk, 6))]
    add("qwen3 attention", [lambda k=k, v=v: X.paged_tree_attention(q, k, v, smap, srow, cu, past, None, D ** -0.5, True, per, max_keys=context + per)
                            for k, v in pools], tot * 8 * D * 4 + T * H * D * 4, 4 * keys * H * D)
    del pools
    # ---- Karuzen's
    gemm_case("karuzen input GEMM (latents fp32 | gate/up + GELU)", n_raw + 2 * FF, W, lambda w: X.gemm_inproj(h, w, raw, n_raw, cat[:, H * D:], True),
              n_raw * 4 + FF * 2, "qwen3 gate/up GEMM + SwiGLU")
    x32 = torch.randn(T, W, device=dev)
    norm = (torch.ones(W, device=dev), torch.zeros(W, device=dev), 0.5)
    gemm_case("karuzen output GEMM (attention | down) + fp32 residual + norm", W, H * D + FF, lambda w: X.gemm_resid32(cat, w, x32, norm=norm, h=h),
              W * 10, "qwen3 down GEMM + residual")
    gemm_case("karuzen query up GEMM", H * D, QR, lambda w: X.gemm(cq, w), H * D * 2, "qwen3 o GEMM + residual")
    lib, p = X.load(), X._p
    lp = [bf(S, R) for _ in range(4)]
    qn, kn = bf(QR), bf(R)
    add("karuzen latent norms + pool scatter", [lambda: X._check(lib.js_latent_post(
        p(raw), n_raw, QR, R, p(qn), p(kn), X.ctypes.c_float(1e-5), p(cq), QR, p(lp[0]), R, S, p(pos), T, p(X.status_word(dev)), 0, X._stream()), "post")],
        T * (QR + R) * 6, 0, 8, "qwen3 head norms + RoPE + KV scatter")
    qa, ol = bf(T, H * R), bf(T, H * R)
    if per < 128:
        gemm_case("karuzen W_uk on the query (batched over heads)", H * R, D, lambda w: X.gemm_batched(q.view(T, H * D), w, qa, H, R, D, D, R, H * R),
                  H * R * 2, "qwen3 o GEMM + residual")
        gemm_case("karuzen W_uv behind the attention (batched over heads)", H * D, R, lambda w: X.gemm_batched(ol, w, cat, H, D, R, R, D, cat.stride(0)),
                  H * (R + D) * 2, "qwen3 o GEMM + residual")
        sp = X.latent_attn_splits(T, H, n_seq, per, R, context + per)
        add(f"karuzen latent attention ({sp} splits)", [lambda l=l: X.latent_attention_rows(
            qa.view(T * H, R), l, H, smap, srow, cu, past, None, D ** -0.5, True, per, out=ol.view(T * H, R), splits=sp) for l in lp],
            tot * R * 2 + T * H * R * 4, 4 * keys * H * R, 8, "qwen3 attention")
    else:
        c, kv = bf(tot, R), bf(tot, 2 * H * D)
        idx = smap.view(-1)
        add("karuzen latent gather", [lambda l=l: X.gather_rows(l, idx, c) for l in lp], tot * R * 4, 0, 8, "qwen3 RMSNorm")
        ws = weights(2 * H * D, R)
        add("karuzen K and V expansion", [lambda w=w: X.gemm(c, w, out=kv) for w in ws],
            (2 * H * D * R + tot * R + 2 * tot * H * D) * 2, 4 * tot * H * D * R, like="qwen3 qkv GEMM")
        kmap, base = torch.arange(tot, dtype=torch.int32, device=dev).view(-1, 1), (srow * (context + per)).contiguous()
        add("karuzen expanded attention", [lambda: X.paged_attention_rows(q, kv[:, :H * D], kv[:, H * D:], kmap, base, cu, past, D ** -0.5, per, cat, context + per)],
            tot * H * D * 4 + T * H * D * 4, 4 * keys * H * D, 4, "qwen3 attention")
    ids, tab = torch.arange(T, dtype=torch.int32, device=dev), bf(32768, W)
    emb = bf(T, W)
    add("karuzen embedding + norm", [lambda: X._check(lib.js_embed_dyt(
        p(ids), p(tab), 32768, W, p(x32), p(emb), p(h), W, p(norm[0]), p(norm[1]), X.ctypes.c_float(0.5), T, W, 0, X._stream()), "embed")],
        T * W * 10, 0, 8, "qwen3 RMSNorm")
    by = {r["kernel"]: r["fraction"] for r in rows}
    for r in rows:
        if r["like"]:
            r["against_like"] = round(by[r["like"]] / max(r["fraction"], 1e-6), 2)       # > 2: more than twice as far from its roofline
    X.check_status(dev)
    return {"rows": T, "sequences": n_seq, "context": context, "peaks": note, "kernels": rows}


def routed_table(T):
    """The routed layers' kernels at Qwen3-30B-A3B sizes (128 experts of 768, 8 a token, width 2048)."""
    from jetspec_b200.ops import cuda_ext as X
    bw, fl, note = peaks()
    E, k, I, W = 128, 8, 768, 2048
    dev = "cuda"
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(torch.bfloat16)
    rows, P = [], T * k
    hit = min(E, P)                          # experts with rows: nearly all of them from a few dozen tokens on
    g = torch.Generator().manual_seed(0)
    idx = torch.stack([torch.randperm(E, generator=g)[:k] for _ in range(T)]).to(torch.int32).to(dev)
    hit = int(idx.unique().numel())
    cnt = torch.bincount(idx.view(-1).long().cpu(), minlength=E)
    off = torch.cat((torch.zeros(1, dtype=torch.long), cnt.cumsum(0))).to(torch.int32).to(dev)
    cover = min(T, ((4 * P // E + 128 + 127) // 128) * 128)
    xs = bf(P, W)

    def add(name, fns, nbytes, flops, inner, like=None):
        us = graph_time_us(fns, inner)
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 4), "like": like})
    gu = [bf(E * 2 * I, W) for _ in range(2)]
    h1, h2, ys = bf(P, I), bf(P, I), bf(P, W)
    add("qwen3 grouped gate/up + SwiGLU", [lambda w=w: X.gemm_grouped(xs, w, h1, P, 2 * I, E, off, cover, X.EPI_SWIGLU) for w in gu],
        hit * 2 * I * W * 2 + P * (W + I) * 2, 4 * P * I * W, 4)
    dn = [bf(E * W, I) for _ in range(3)]
    add("qwen3 grouped down (the same kernel in both)", [lambda w=w: X.gemm_grouped(h1, w, ys, P, W, E, off, cover, X.EPI_STORE) for w in dn],
        hit * I * W * 2 + P * (W + I) * 2, 2 * P * I * W, 6)
    del gu
    up = [bf(E * I, W) for _ in range(3)]
    add("karuzen grouped up + relu^2", [lambda w=w: X.gemm_grouped(xs, w, h2, P, I, E, off, cover, X.EPI_RELU2) for w in up],
        hit * I * W * 2 + P * (W + I) * 2, 2 * P * I * W, 6, "qwen3 grouped down (the same kernel in both)")
    z = torch.randn(T, E + 128, device=dev)
    corr, act = torch.randn(E, device=dev), bf(T, I)
    wts, ix = torch.empty(T, k, device=dev), torch.empty(T, k, dtype=torch.int32, device=dev)
    zz = z[:, :E].contiguous()
    add("qwen3 softmax router", [lambda: X.moe_route(zz, k, True)], T * E * 4, 0, 8)
    add("karuzen sigmoid router + shared gate", [lambda: X.sigmoid_route(z, corr, k, 2.5, E, act, wts=wts, idx=ix)], T * (E * 4 + I * 4), 0, 8, "qwen3 softmax router")
    lib, p = X.load(), X._p
    inv, rw = torch.randperm(P, device=dev).to(torch.int32), torch.rand(P, device=dev)
    order = torch.randperm(P, device=dev).to(torch.int32)
    res = bf(T, W)
    add("qwen3 combine + residual (invert + sum)", [lambda: X._check(lib.js_moe_combine(
        p(ys), W, p(order), p(rw), T, k, W, p(inv), p(res), p(res), W, 0, X._stream()), "combine")], P * W * 2 + T * W * 4, 0, 8)
    x32, h, one = torch.randn(T, W, device=dev), bf(T, W), torch.ones(W, device=dev)
    add("karuzen combine + fp32 residual + norm", [lambda: X._check(lib.js_combine_dyt(
        p(ys), W, p(inv), p(rw), k, None, p(x32), p(h), W, p(one), p(one), X.ctypes.c_float(0.5), T, W, 0, X._stream()), "combine")],
        P * W * 2 + T * W * 10, 0, 8, "qwen3 combine + residual (invert + sum)")
    by = {r["kernel"]: r["fraction"] for r in rows}
    for r in rows:
        if r["like"]:
            r["against_like"] = round(by[r["like"]] / max(r["fraction"], 1e-6), 2)
    X.check_status(dev)
    return {"rows": T, "experts": E, "peaks": note, "kernels": rows}


def main(part: str = "all", depth: int = 8) -> None:
    assert torch.cuda.is_available(), "this bench needs a GPU"
    if part in ("all", "kernels"):
        for args in ((1, 2048, 1), (16, 2048, 16), (128, 2048, 16), (2048, 0, 1)):
            print(json.dumps({"bench": "karuzen kernels", **kernel_table(*args)}), flush=True)
            torch.cuda.empty_cache()
        for T in (16, 2048):
            print(json.dumps({"bench": "karuzen routed kernels", **routed_table(T)}), flush=True)
            torch.cuda.empty_cache()
    if part in ("all", "models"):
        for name, cfgs in pairs(depth).items():
            for cfg in cfgs:
                print(json.dumps({"bench": "karuzen throughput", "data": "synthetic", "dtype": "bf16", **throughput(name, cfg)}), flush=True)


if __name__ == "__main__":
    main(*sys.argv[1:2])
