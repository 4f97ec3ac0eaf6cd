"""Prefill and decode throughput of Kizezen beside Qwen3 and Karuzen of equal size, and the roofline of every kernel of a layer.

    python bench.py --design kizezen                 # what this module's main() runs
    python bench.py --design kizezen --part kernels  # per-kernel timings only

Methods, peaks and the form of the tables are those of ``bench/latent_tps.py``.  Models: random weights, the same width,
depth, vocabulary and feed-forward parameters (Kizezen's has two matrices, so its width is half as much again).  The like
kernels are those of the framework's closest model: Qwen3's GEMMs, norms and attention, Karuzen's latent attention,
Zasipel's delta rule for the retention (recurrences with a state of the same size).
"""
from __future__ import annotations

import json
import os
import sys

import torch

# `bench` as a module name is bench.py beside this folder, so the scripts in it import each other by their own names
sys.path[:0] = [os.path.dirname(os.path.dirname(os.path.abspath(__file__))), os.path.dirname(os.path.abspath(__file__))]

import latent_tps  # noqa: E402
from latent_tps import graph_time_us, peaks, throughput  # noqa: E402


def mixers(heads, kv, window=1024, kv_rank=512):
    """One mixer of each kind for a model of ``heads`` 128-wide heads."""
    from jetspec_b200.models import BandScaling, LatentAttentionConfig, RampScaling, RetentionConfig, RotaryConfig, WindowAttentionConfig
    win = WindowAttentionConfig(heads, kv, 128, 128, window, 128, 5e5, 128 ** -0.5, sink=False, qk_norm=False, bias=True, keep_first=4,
                                sink_logits=True, proj_norm=True, o_bias=False, gate=True,
                                rot=RotaryConfig(128, 5e5, "half", BandScaling(8.0, 1.0, 4.0, 8192)))
    lat = LatentAttentionConfig(heads, 96, 128, 0, kv_rank, 128 ** -0.5, rot=RotaryConfig(32, 1e4, "next", RampScaling(40.0, 4096, 32.0, 1.0)),
                                sink_logits=True, gate=True)
    n = heads // 2
    ret = RetentionConfig(n, 128, 256, [1.0 - 2.0 ** (-5 - 7 * i / max(1, n - 1)) for i in range(n)], RotaryConfig(128, 1e4))
    return ret, win, lat


def pairs(depth: int):
    """name -> configurations of equal size; Kizezen's layers repeat (retention, window, latent, window)."""
    from jetspec_b200.models import KizezenConfig, KizezenLayerConfig
    other = latent_tps.pairs(depth)
    out = {}
    for name, width, heads, kv, ff in (("dense 4096", 4096, 32, 8, 12288), ("dense 2048", 2048, 16, 8, 6144)):
        ret, win, lat = mixers(heads, kv)
        layers = [KizezenLayerConfig((ret, win, lat, win)[i % 4], ff * 3 // 2) for i in range(depth)]
        out[name] = (KizezenConfig(vocab_size=32768, hidden_size=width, layers=layers), *reversed(other[name]))
    return out


def kernel_table(T, context, n_seq):
    """Per-launch times of the layers' kernels for ``T`` rows (``n_seq`` sequences with ``context`` cached tokens each) at width
    4096, 32 heads (window attention over 8 key heads, latents of 512 + 32, retention 16 x 128 x 256), window 1024."""
    from jetspec_b200.models import DeltaConfig
    from jetspec_b200.ops import cuda_ext as X
    bw, fl, note = peaks()
    W, H, KV, D, WIN, KEEP, FF, dev = 4096, 32, 8, 128, 1024, 4, 12288, "cuda"
    ret, win, lat = mixers(H, KV, WIN)
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(torch.bfloat16)
    i32 = dict(dtype=torch.int32, device=dev)
    rows = []
    lib, p = X.load(), X._p

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
    # ---- Qwen3's kernels at this width
    h, nw, qkv, xr = bf(T, W), bf(W), bf(T, 6144), bf(T, W)
    att, act = bf(T, W), bf(T, FF)
    gemm_case("qwen3 qkv GEMM", 6144, W, lambda w: X.gemm(h, w), 6144 * 2)
    gemm_case("qwen3 o GEMM + residual", W, W, lambda w: X.gemm(att, w, out=xr, residual=xr), W * 4)
    if T >= 1024:
        gemm_case("qwen3 gate/up GEMM + SwiGLU", 2 * FF, W, lambda w: X.gemm(h, w, epi=X.EPI_SWIGLU, bn=256, split=1, deep=0), FF * 2)
    else:
        gemm_case("qwen3 gate/up GEMM + SwiGLU", 2 * FF, W, lambda w: X.gemm(h, w, epi=X.EPI_SWIGLU), FF * 2)
    gemm_case("qwen3 down GEMM + residual", W, FF, lambda w: X.gemm(act, w, out=xr, residual=xr), W * 4)
    add("qwen3 RMSNorm", [lambda: X.rmsnorm(h, nw, 1e-6)], T * W * 4, 0, 8)
    q, freq = bf(T, H, D), X.inv_freq(D, 1e6, dev)
    kp, vp = bf(KV, S, D), bf(KV, S, D)
    add("qwen3 head norms + RoPE + KV scatter", [lambda: X.qkv_post(qkv, nw[:D], nw[:D], pos, pos, freq, q, kp, vp, H, KV, 1e-6)], T * 6144 * 4, 0, 8)
    keys = n_seq * per * context + n_seq * per * (per + 1) // 2
    pools = [(bf(KV, S, D), bf(KV, S, D)) for _ in range(max(1, min(6, int(300e6 / (tot * 4096)) + 1)))]
    add("qwen3 attention", [lambda k=k, v=v: X.paged_tree_attention(q, k, v, smap, srow, cu, past, None, D ** -0.5, True, per, max_keys=context + per)
                            for k, v in pools], tot * KV * D * 4 + T * H * D * 4, 4 * keys * H * D)
    # ---- Kizezen: window attention
    raw, a_w = torch.randn(T, 640, device=dev), bf(T, 12288)
    gemm_case("kizezen input GEMM, window attention (gates fp32 | q k v)", 128 + 6144, W,
              lambda w: X.gemm_inproj(h, w, raw, 128, qkv, False, act=X.ACT_NONE), 512 + 6144 * 2, "qwen3 qkv GEMM")
    bias, qn, kn = torch.randn(6144, device=dev), torch.ones(H * D, device=dev), torch.ones(KV * D, device=dev)
    table = torch.randn(T, 144, 2, device=dev)
    wq, wo = bf(T, H * D), bf(T, H * D)
    add("kizezen bias + projection norms + rotation + KV scatter", [lambda: X._check(lib.js_attn_post(
        p(qkv), 6144, p(bias), p(qn), p(kn), H, KV, H // KV, D, D, D, D, D, D, 0, p(table), 144, X.ctypes.c_float(1e-5), p(pos), S, T, p(wq), p(kp), p(vp),
        status, 0, X._stream()), "post")], T * 6144 * 4, 0, 8, "qwen3 head norms + RoPE + KV scatter")
    seen_w = n_seq * sum(min(WIN + KEEP, context + i + 1) for i in range(per))
    keys_w = n_seq * min(context + per, WIN + KEEP + per - 1)
    sp = X.window_attn_splits(T, H, KV, context + per, WIN, KEEP, seqs=n_seq)
    ws = {"o": torch.zeros(sp, T, H, D, device=dev), "ml": torch.zeros(sp, T, H, 2, device=dev)}
    sinks, gate = torch.randn(H, device=dev), torch.randn(T, 128, device=dev)
    add(f"kizezen window attention, sinks, gate ({sp} splits)", [lambda k=k, v=v: X.window_attention_tc(
        wq.view(T, H, D), k, v, smap, srow, cu, past, None, D ** -0.5, WIN, sinks, True, wo, splits=sp, ws=ws, keep_first=KEEP, gate=gate) for k, v in pools],
        keys_w * KV * D * 4 + T * H * D * 4, 4 * seen_w * H * D, like="qwen3 attention")
    del pools
    # ---- latent attention, beside Karuzen's
    R, E = lat.kv_rank, lat.rot_dim
    RP, QR = (R + E + 63) // 64 * 64, 1536
    gemm_case("kizezen input GEMM, latent attention (row and gates fp32 | q)", 640 + H * D, W,
              lambda w: X.gemm_inproj(h, w, raw, 640, wq, False, act=X.ACT_NONE), 2560 + H * D * 2, "qwen3 qkv GEMM")
    lp, lk = [bf(S, RP) for _ in range(4)], [bf(S, R) for _ in range(4)]
    ln, kqn, kkn, rawk, cq = torch.ones(R, device=dev), bf(QR), bf(R), torch.randn(T, QR + R, device=dev), bf(T, QR)
    add("karuzen latent norms + pool scatter", [lambda: X._check(lib.js_latent_post(
        p(rawk), QR + R, QR, R, p(kqn), p(kkn), X.ctypes.c_float(1e-5), p(cq), QR, p(lk[0]), R, S, p(pos), T, status, 0, X._stream()), "post")],
        T * (QR + R) * 6, 0, 8)
    add("kizezen latent norm + rotations + pool scatter", [lambda: X._check(lib.js_latent_rot_post(
        p(raw), 640, R, E, p(ln), X.ctypes.c_float(1e-5), p(lp[0]), RP, S, p(pos), p(wq), H * D, H, D, lat.dim, p(table), 144, T, status, 0, X._stream()),
        "post")], T * ((R + E) * 6 + H * E * 4), 0, 8, "karuzen latent norms + pool scatter")
    if per < 128:
        for fam, rp, vk, pool, kw in (("karuzen", R, R, lk, {}), ("kizezen", RP, R, lp, dict(out_cols=R, sinks=sinks, gate=gate))):
            like = (lambda s: s) if fam == "kizezen" else (lambda s: None)
            qa, ol = bf(T, H * rp), bf(T, H * rp)
            gemm_case(f"{fam} W_uk on the query (batched over heads)", H * rp, D, lambda w: X.gemm_batched(wq, w, qa, H, rp, D, D, rp, H * rp),
                      H * rp * 2, like("karuzen W_uk on the query (batched over heads)"))
            gemm_case(f"{fam} W_uv behind the attention (batched over heads)", H * D, vk,
                      lambda w: X.gemm_batched(ol, w, wo, H, D, vk, rp, D, H * D), H * D * 2 + H * vk * 2 - vk * 2,
                      like("karuzen W_uv behind the attention (batched over heads)"))
            sp = X.latent_attn_splits(T, H, n_seq, per, rp, context + per, vk)
            add(f"{fam} latent attention", [lambda l=l: X.latent_attention_rows(
                qa.view(T * H, rp), l, H, smap, srow, cu, past, None, D ** -0.5, True, per, out=ol.view(T * H, rp), splits=sp, **kw) for l in pool],
                tot * rp * 2 + T * H * (rp + vk) * 2, 2 * keys * H * (rp + vk), 8, like("karuzen latent attention"))
    else:
        kv, idx = bf(tot, 2 * H * D), smap.view(-1)
        kmap, base = torch.arange(tot, **i32).view(-1, 1), (srow * (context + per)).contiguous()
        for fam, rp, pool, kw in (("karuzen", R, lk, {}), ("kizezen", RP, lp, dict(sinks=sinks, gate=gate))):
            like = (lambda s: s) if fam == "kizezen" else (lambda s: None)
            c = bf(tot, rp)
            add(f"{fam} latent gather", [lambda l=l: X.gather_rows(l, idx, c) for l in pool], tot * rp * 4, 0, 8, like("karuzen latent gather"))
            wts = [bf(2 * H * D, rp) for _ in range(24)]
            add(f"{fam} K and V expansion", [lambda w=w: X.gemm(c, w, out=kv) for w in wts], (2 * H * D * rp + tot * rp + 2 * tot * H * D) * 2,
                4 * tot * H * D * rp, like=like("karuzen K and V expansion"))
            add(f"{fam} expanded attention", [lambda: X.paged_attention_rows(
                wq.view(T, H, D), kv[:, :H * D], kv[:, H * D:], kmap, base, cu, past, D ** -0.5, per, wo, context + per, **kw)],
                tot * H * D * 4 + T * H * D * 4, 4 * keys * H * D, 4, like("karuzen expanded attention"))
    # ---- retention, beside Zasipel's delta rule with a state of the same size
    gemm_case("kizezen input GEMM, retention (q k v gate)", 12288, W, lambda w: X.gemm_inproj(h, w, None, 0, a_w, False, act=X.ACT_NONE),
              12288 * 2, "qwen3 qkv GEMM")
    a_w.copy_(bf(T, 12288) * 30)
    dc = DeltaConfig(32, 16, D, D, 4)
    pre, dg, z, b = bf(T, dc.channels) * 30, bf(T, 4096), torch.randn(T, 32, device=dev), torch.randn(T, 32, device=dev)
    taps, A, dt, on, do = bf(dc.channels, 4), torch.linspace(-4, 0, 32, device=dev).to(torch.bfloat16), bf(32) - 2, bf(D), bf(T, 4096)
    sbytes = n_seq * 16 * 128 * 256 * 4
    copies = max(1, min(8, int(300e6 / sbytes) + 1))
    st = [(torch.zeros(n_seq + 1, 32, D, D, device=dev), bf(n_seq + 1, 4, dc.channels)) for _ in range(copies)]
    add("zasipel delta rule, head decay (all kernels between the GEMMs)",
        [lambda s=s: X.delta_forward(dc, pre, z, b, taps, A, dt, s[0], s[1], srow, cu, past, dg, on, "silu", 1e-6, do, max_rows=per) for s in st],
        T * (dc.channels + 2 * 4096) * 2 + T * 64 * 4 + 2 * sbytes, 7 * T * 32 * D * D)
    st = [torch.zeros(n_seq + 1, 16, 128, 256, device=dev) for _ in range(copies)]
    add("kizezen retention (all kernels between the GEMMs)",
        [lambda s=s: X.retention_forward(ret, a_w, (2048, 4096, 8192), table, s, srow, cu, past, None, 1e-5, do, per) for s in st],
        T * (12288 + 4096) * 2 + T * 64 * 8 + 2 * sbytes, 4 * T * 16 * 128 * 256, like="zasipel delta rule, head decay (all kernels between the GEMMs)")
    del st
    # ---- output, feed-forward, norms
    x32, w1, up, hh = torch.randn(T, W, device=dev), torch.ones(W, device=dev), bf(T, FF * 3 // 2), bf(T, W)
    gemm_case("kizezen output GEMM + fp32 residual", W, H * D, lambda w: X.gemm_resid32(wo, w, x32), W * 8, "qwen3 o GEMM + residual")
    gemm_case("kizezen up GEMM + exact gelu", FF * 3 // 2, W, lambda w: X.gemm_inproj(h, w, None, 0, up, False, act=X.ACT_GELU_ERF), FF * 3,
              "qwen3 gate/up GEMM + SwiGLU")
    gemm_case("kizezen down GEMM + fp32 residual", W, FF * 3 // 2, lambda w: X.gemm_resid32(up, w, x32), W * 8, "qwen3 down GEMM + residual")
    add("kizezen norm of the fp32 stream", [lambda: X._check(lib.js_rms_rows(
        p(x32), p(w1), X.ctypes.c_float(1e-5), p(hh), W, T, W, None, 0, 0, X._stream()), "norm")], T * W * 6, 0, 8, "qwen3 RMSNorm")
    ids, tab, fr = torch.arange(T, **i32), bf(32768, W), torch.rand(144, device=dev)
    add("kizezen embedding + norm + rotary tables", [lambda: X._check(lib.js_embed_rms(
        p(ids), p(tab), 32768, W, X.ctypes.c_float(1.0), p(w1), X.ctypes.c_float(1e-5), p(x32), p(hh), W, T, W, p(pos), None, 0, p(fr), p(fr), 144, p(table), 0,
        X._stream()), "embed")], T * W * 8 + T * 144 * 8, 0, 8, "qwen3 RMSNorm")
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
            print(json.dumps({"bench": "kizezen kernels", **kernel_table(*args)}), flush=True)
            torch.cuda.empty_cache()
    if part in ("all", "models"):
        for name, cfgs in pairs(depth).items():
            for cfg in cfgs:
                print(json.dumps({"bench": "kizezen throughput", "data": "synthetic", "dtype": "bf16", **throughput(name, cfg)}), flush=True)


if __name__ == "__main__":
    main(*sys.argv[1:2])
