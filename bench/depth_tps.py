"""Prefill and decode throughput of Sogidra beside Kizezen and Qwen3 of equal size, and the roofline of every kernel of a layer.

    python bench.py --design sogidra                 # what this module's main() runs
    python bench.py --design sogidra --part kernels  # per-kernel timings only

Methods, peaks and the form of the tables are those of ``bench/latent_tps.py``.  Models: random weights, the same width, depth,
vocabulary, key and value heads and feed-forward parameters.  The like kernels are those of the framework's closest models:
Kizezen's window attention, norms and embedding, Qwen3's GEMMs, full attention and the step behind its projections.
"""
from __future__ import annotations

import json
import os
import sys

import torch

# `bench` as a module name is bench.py beside this folder, so the scripts in it import each other by their own names
sys.path[:0] = [os.path.dirname(os.path.dirname(os.path.abspath(__file__))), os.path.dirname(os.path.abspath(__file__))]

import mixed_tps  # noqa: E402
from latent_tps import graph_time_us, peaks, throughput  # noqa: E402

POOL, CAP = 16, 50.0


def mixers(heads, kv, window=1024):
    """Window attention with pooled blocks (128-wide heads) and differential attention (two maps of 64 over 128-wide values)."""
    from jetspec_b200.models import WindowAttentionConfig
    common = dict(rot_dims=0, rot_base=1.0, sink=False, o_bias=False)
    pooled = WindowAttentionConfig(heads, kv, 128, 128, window, scale=128 ** -0.5, qk_norm=True, bias=False, tie_values=True, softcap=CAP, pool=POOL, **common)
    diff = lambda src=None: WindowAttentionConfig(heads, kv, 64, 128, 0, scale=64 ** -0.5, qk_norm=False, bias=True, diff=0.4, temp_every=1024,
                                                  temp_coef=0.5, kv_from=src, **common)
    return pooled, diff


def pairs(depth: int):
    """name -> configurations of equal size; Sogidra's layers repeat (pooled, differential, pooled, differential on the second
    layer's keys)."""
    from jetspec_b200.models import SogidraConfig, SogidraLayerConfig
    other = mixed_tps.pairs(depth)
    out = {}
    for name, width, heads, kv, ff in (("dense 4096", 4096, 32, 8, 12288), ("dense 2048", 2048, 16, 8, 6144)):
        pooled, diff = mixers(heads, kv)
        layers = [SogidraLayerConfig((pooled, diff(), pooled, diff(i // 4 * 4 + 1))[i % 4], ff * 3 // 2) for i in range(depth)]
        cfg = SogidraConfig(vocab_size=32768, hidden_size=width, layers=layers, max_positions=4096)
        kizezen, qwen = other[name][:2]
        out[name] = (cfg, kizezen, qwen)
    return out


def kernel_table(T, context, n_seq):
    """Per-launch times of the layers' kernels for ``T`` rows (``n_seq`` sequences with ``context`` cached tokens each) at width
    4096, 32 heads over 8, window 1024, blocks of 16."""
    from jetspec_b200.ops import cuda_ext as X
    bw, fl, note = peaks()
    W, H, KV, D, WIN, KEEP, FF, dev = 4096, 32, 8, 128, 1024, 4, 12288, "cuda"
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(torch.bfloat16)
    i32 = dict(dtype=torch.int32, device=dev)
    rows = []
    lib, p, f = X.load(), X._p, X.ctypes.c_float

    def add(name, fns, nbytes, flops, inner=None, like=None):
        us = graph_time_us(fns, inner or 2 * len(fns))
        roof = max(nbytes / bw, flops / fl) * 1e6
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 6), "like": like})

    def gemm_case(name, n, k, call, out_bytes, like=None):
        ws = [bf(n, k) for _ in range(min(24, max(2, int(400e6 / (n * k * 2)) + 1)))]
        add(name, [lambda w=w: call(w) for w in ws], (n * k + T * k) * 2 + T * out_bytes, 2 * T * n * k, like=like)

    per = T // n_seq
    tot, S = n_seq * (context + per), n_seq * (context + per) + 64
    smap = torch.randperm(S, device=dev).to(torch.int32)[:tot].view(n_seq, context + per).contiguous()
    srow = torch.arange(n_seq, **i32)
    cu = (torch.arange(n_seq + 1, **i32) * per).contiguous()
    past = torch.full((n_seq,), context, **i32)
    pos = torch.arange(T, **i32)
    status = p(X.status_word(dev))
    # ---- Qwen3's and Kizezen's kernels at this width
    h, nw, qkv, xr = bf(T, W), bf(W), bf(T, 6144), bf(T, W)
    att, act = bf(T, W), bf(T, FF)
    gemm_case("qwen3 qkv GEMM", 6144, W, lambda w: X.gemm(h, w), 6144 * 2)
    gemm_case("qwen3 o GEMM + residual", W, W, lambda w: X.gemm(att, w, out=xr, residual=xr), W * 4)
    if T >= 1024:
        gemm_case("qwen3 gate/up GEMM + SwiGLU", 2 * FF, W, lambda w: X.gemm(h, w, epi=X.EPI_SWIGLU, bn=256, split=1, deep=0), FF * 2)
    else:
        gemm_case("qwen3 gate/up GEMM + SwiGLU", 2 * FF, W, lambda w: X.gemm(h, w, epi=X.EPI_SWIGLU), FF * 2)
    gemm_case("qwen3 down GEMM + residual", W, FF, lambda w: X.gemm(act, w, out=xr, residual=xr), W * 4)
    q, freq = bf(T, H, D), X.inv_freq(D, 1e6, dev)
    kp, vp = bf(KV, S, D), bf(KV, S, D)
    add("qwen3 head norms + RoPE + KV scatter", [lambda: X.qkv_post(qkv, nw[:D], nw[:D], pos, pos, freq, q, kp, vp, H, KV, 1e-6)], T * 6144 * 4, 0, 8)
    keys = n_seq * per * context + n_seq * per * (per + 1) // 2
    pools = [(bf(KV, S, D), bf(KV, S, D)) for _ in range(max(1, min(6, int(300e6 / (tot * 4096)) + 1)))]
    add("qwen3 attention", [lambda k=k, v=v: X.paged_tree_attention(q, k, v, smap, srow, cu, past, None, D ** -0.5, True, per, max_keys=context + per)
                            for k, v in pools], tot * KV * D * 4 + T * H * D * 4, 4 * keys * H * D)
    wq, wo = bf(T, H * D), bf(T, H * D)

    def split_space(sp, maps=1):
        return {"o": torch.zeros(sp, T, H * maps, D, device=dev), "ml": torch.zeros(sp, T, H * maps, 2, device=dev)}
    seen = lambda keep: n_seq * sum(min(WIN + keep, context + i + 1) for i in range(per))
    span = lambda keep: n_seq * min(context + per, WIN + keep + per - 1)
    sp = X.window_attn_splits(T, H, KV, context + per, WIN, KEEP, seqs=n_seq)
    ws, sinks, gate = split_space(sp), torch.randn(H, device=dev), torch.randn(T, 128, device=dev)
    add("kizezen window attention, sinks, gate", [lambda k=k, v=v: X.window_attention_tc(
        wq.view(T, H, D), k, v, smap, srow, cu, past, None, D ** -0.5, WIN, sinks, True, wo, splits=sp, ws=ws, keep_first=KEEP, gate=gate) for k, v in pools],
        span(KEEP) * KV * D * 4 + T * H * D * 4, 4 * seen(KEEP) * H * D)
    x32, w1, hh, y, fr, table = torch.randn(T, W, device=dev), torch.ones(W, device=dev), bf(T, W), bf(T, W), torch.rand(144, device=dev), torch.randn(T, 144, 2, device=dev)
    add("kizezen norm of the fp32 stream", [lambda: X._check(lib.js_rms_rows(
        p(x32), p(w1), f(1e-5), p(hh), W, T, W, None, 0, 0, X._stream()), "norm")], T * W * 6, 0, 8)
    ids, tab, ptab = torch.arange(T, **i32), bf(32768, W), bf(4096, W)
    embed = lambda pt, n: X._check(lib.js_embed_rms(p(ids), p(tab), 32768, W, f(1.0), p(w1), f(1e-5), p(x32), p(hh), W, T, W, p(pos), pt, n, p(fr), p(fr), 2,
                                                    p(table), 0, X._stream()), "embed")
    add("kizezen embedding + norm", [lambda: embed(None, 0)], T * W * 8, 0, 8)
    # ---- pooled window attention
    gemm_case("input GEMM, pooled attention (q k)", 5120, W, lambda w: X.gemm_inproj(h, w, None, 0, qkv[:, :5120], False, act=X.ACT_NONE), 5120 * 2, "qwen3 qkv GEMM")
    pfreq, bias = X.pair_freq(0, 1.0, dev), torch.randn(6144, device=dev)

    def post(maps, d, norm, every, vcol, b):
        return lambda: X._check(lib.js_window_post(
            p(qkv), 6144, p(b), H, KV, H // KV, maps, d, D, 128 // maps, D, D, 0, p(pfreq), norm, f(1e-5), every, f(0.5), vcol, 1, p(pos), p(pos), S, T, p(wq),
            p(kp), p(vp), status, 0, X._stream()), "post")
    add("norms + KV scatter, values from keys", [post(1, D, 1, 0, H * D, None)], T * (5120 + H * D + 2 * KV * D) * 2, 0, 8, "qwen3 head norms + RoPE + KV scatter")
    nb = (context + per) // POOL
    kb, vb = bf(KV, n_seq * (nb + 1), D), bf(KV, n_seq * (nb + 1), D)
    bmap = torch.randperm(n_seq * (nb + 1), device=dev).to(torch.int32).view(n_seq, nb + 1).contiguous()
    ends = n_seq * ((context + per) // POOL - context // POOL)
    add("block means", [lambda k=k, v=v: X.pool_blocks(k, v, kb, vb, bmap, POOL, smap, srow, cu, past, rows=T) for k, v in pools],
        ends * KV * D * 4 * (POOL + 1), 0, like="qwen3 head norms + RoPE + KV scatter" if ends else None)
    sp1 = X.window_attn_splits(T, H, KV, context + per, WIN, 0, POOL, n_seq)
    ws1 = split_space(sp1)
    far = n_seq * sum(max(0, context + i + 1 - WIN) // POOL for i in range(per))
    far_span = n_seq * (max(0, context + per - WIN) // POOL)
    add(f"pooled window attention, capped ({sp1} splits)", [lambda k=k, v=v: X.window_attention_tc(
        wq.view(T, H, D), k, v, smap, srow, cu, past, None, D ** -0.5, WIN, False, True, wo, splits=sp1, ws=ws1, softcap=CAP,
        blocks=(kb, vb, bmap, POOL)) for k, v in pools],
        (span(0) + far_span) * KV * D * 4 + T * H * D * 4, 4 * (seen(0) + far) * H * D, like="kizezen window attention, sinks, gate")
    # ---- differential attention
    gemm_case("input GEMM, differential attention (q k v)", 6144, W, lambda w: X.gemm_inproj(h, w, None, 0, qkv, False, act=X.ACT_NONE), 6144 * 2, "qwen3 qkv GEMM")
    gemm_case("input GEMM, differential attention over another layer's keys (q)", H * D, W, lambda w: X.gemm_inproj(h, w, None, 0, wq, False, act=X.ACT_NONE),
              H * D * 2, "qwen3 qkv GEMM")
    add("bias + temperature + KV scatter", [post(2, 64, 0, 1024, (H + KV) * D, bias)], T * 6144 * 4, 0, 8, "qwen3 head norms + RoPE + KV scatter")
    sp2 = X.window_attn_splits(T, H, KV, context + per, 0, seqs=n_seq)
    ws2, lam = split_space(sp2, 2), torch.tensor([0.5], device=dev)
    add(f"differential attention ({sp2} splits)", [lambda k=k, v=v: X.window_attention_tc(
        wq.view(T, H, D), k, v, smap, srow, cu, past, None, 0.125, 0, False, True, wo, splits=sp2, ws=ws2, diff=(lam, 0.6, 1e-5)) for k, v in pools],
        tot * KV * D * 4 + T * H * D * 4, 6 * keys * H * D, like="qwen3 attention")
    del pools
    # ---- output, feed-forward, residual steps
    up, x2 = bf(T, FF * 3 // 2), torch.randn(T, W, device=dev)
    gemm_case("output GEMM", W, H * D, lambda w: X.gemm(wo, w, out=y), W * 2, "qwen3 o GEMM + residual")
    gemm_case("up GEMM + xIELU", FF * 3 // 2, W, lambda w: X.gemm_inproj(h, w, None, 0, up, False, act=X.ACT_XIELU, act_args=(0.9, 1.1)), FF * 3,
              "qwen3 gate/up GEMM + SwiGLU")
    gemm_case("down GEMM", W, FF * 3 // 2, lambda w: X.gemm(up, w, out=y), W * 2, "qwen3 down GEMM + residual")
    add("residual step within a layer (output norm, sum, next norm)", [lambda: X.sandwich(y, x32, w1, x2, w1, 1e-5, hh, W)], T * W * 12, 0, 8,
        "kizezen norm of the fp32 stream")
    hist = torch.randn(9, T, W, device=dev)
    for n in (1, 4, 8):
        d = torch.rand(n + 1, device=dev)
        add(f"residual step at the end of layer {n} (the same, depth average over {n + 1})",
            [lambda: X.sandwich(y, x32, w1, x2, w1, 1e-5, hh, W, hist=hist, d=d)], T * W * (16 + 4 * n), 0, 8, "kizezen norm of the fp32 stream")
    add("embedding + positions + norm", [lambda: embed(p(ptab), 4096)], T * W * 10, 0, 8, "kizezen embedding + norm")
    by = {r["kernel"]: r["fraction"] for r in rows}
    for r in rows:
        if r["like"]:
            r["against_like"] = round(by[r["like"]] / max(r["fraction"], 1e-9), 2)       # > 2: more than twice as far from its roofline
    X.check_status(dev)
    return {"rows": T, "sequences": n_seq, "context": context, "peaks": note, "kernels": rows}


def main(part: str = "all", depth: int = 8) -> None:
    assert torch.cuda.is_available(), "this bench needs a GPU"
    if part in ("all", "kernels"):
        for args in ((1, 2048, 1), (16, 2048, 16), (2048, 0, 1)):
            print(json.dumps({"bench": "sogidra kernels", **kernel_table(*args)}), flush=True)
            torch.cuda.empty_cache()
    if part in ("all", "models"):
        for name, cfgs in pairs(depth).items():
            for cfg in cfgs:
                print(json.dumps({"bench": "sogidra throughput", "data": "synthetic", "dtype": "bf16", **throughput(name, cfg)}), flush=True)


if __name__ == "__main__":
    main(*sys.argv[1:2])
