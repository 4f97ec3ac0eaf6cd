"""Prefill and decode throughput of Zasipel beside Qwen3-MoE of equal size, and the roofline of every kernel of a layer.

    python bench.py --design zasipel                 # what this module's main() runs
    python bench.py --design zasipel --part kernels  # per-kernel timings only

Methods, peaks and the form of the tables are those of ``bench/latent_tps.py``.  Models: random weights, the same width,
depth, vocabulary, experts and mixer width (window heads + delta heads = attention heads); Zasipel also runs a shared
expert.  The like kernel of the recurrence is the attention: both mix over time.
"""
from __future__ import annotations

import json
import os
import sys

import torch

# `bench` as a module name is bench.py beside this folder, so the scripts in it import each other by their own names
sys.path[:0] = [os.path.dirname(os.path.dirname(os.path.abspath(__file__))), os.path.dirname(os.path.abspath(__file__))]

from latent_tps import graph_time_us, peaks, throughput  # noqa: E402


def pairs(depth: int):
    """name -> (Zasipel config, Qwen3-MoE config) of equal size.  Every fourth Zasipel layer is a channel-decay layer."""
    from jetspec_b200.models import (DeltaConfig, Qwen3Config, TableExpertsConfig, WindowAttentionConfig, ZasipelConfig,
                                     ZasipelLayerConfig)

    def za(width, heads, kv, experts, top, ff, vocab, window=1024):
        win = WindowAttentionConfig(heads // 2, kv, 128, 128, window, 64, 1e6, 128 ** -0.5)
        head = DeltaConfig(heads // 2, heads // 4, 128, 128, 4)
        chan = DeltaConfig(heads, heads, 128, 128, 4, decay="channel", gate="sigmoid", decay_rank=128, gate_rank=128)
        moe = TableExpertsConfig(experts, top, ff, ff)
        layers = [ZasipelLayerConfig(chan, None, moe) if i % 4 == 3 else ZasipelLayerConfig(head, win, moe) for i in range(depth)]
        return ZasipelConfig(vocab_size=vocab, hidden_size=width, layers=layers)

    def qw(width, heads, kv, experts, top, ff, vocab):
        return Qwen3Config(vocab_size=vocab, hidden_size=width, intermediate_size=3 * width, num_hidden_layers=depth,
                           num_attention_heads=heads, num_key_value_heads=kv, head_dim=128, num_experts=experts,
                           num_experts_per_tok=top, moe_intermediate_size=ff, model_type="qwen3_moe")
    return {"2048, 128 experts of 768, 8 a token": (za(2048, 32, 4, 128, 8, 768, 32768), qw(2048, 32, 4, 128, 8, 768, 32768)),
            "4096, 16 experts of 1536, 4 a token": (za(4096, 32, 8, 16, 4, 1536, 32768), qw(4096, 32, 8, 16, 4, 1536, 32768))}


def kernel_table(T, context, n_seq):
    """Per-launch times of a layer's kernels for ``T`` rows (``n_seq`` sequences with ``context`` cached tokens each) at
    width 2048, 16 window heads over 4, 16 delta heads over 8 (channel decay: 32), head size 128, window 1024."""
    from jetspec_b200.models import DeltaConfig
    from jetspec_b200.ops import cuda_ext as X
    bw, fl, note = peaks()
    W, D, WIN, dev = 2048, 128, 1024, "cuda"
    bf = lambda *s: (torch.randn(*s, device=dev) * 0.02).to(torch.bfloat16)
    i32 = dict(dtype=torch.int32, device=dev)
    rows = []

    def add(name, fns, nbytes, flops, inner=None, like=None, rate=None):
        us = graph_time_us(fns, inner or 2 * len(fns))
        roof = max(nbytes / bw, flops / (rate or fl)) * 1e6
        rows.append({"kernel": name, "us": round(us, 2), "roofline_us": round(roof, 2), "fraction": round(roof / us, 4), "like": like})

    def gemm_case(name, n, k, call, out_bytes, like=None):
        ws = [bf(n, k) for _ in range(min(24, max(2, int(400e6 / (n * k * 2)) + 1)))]
        add(name, [lambda w=w: call(w) for w in ws], (n * k + T * k) * 2 + T * out_bytes, 2 * T * n * k, like=like)

    per = T // n_seq
    S = n_seq * (context + per) + 64
    smap = torch.randperm(S, device=dev).to(torch.int32)[: n_seq * (context + per)].view(n_seq, context + per).contiguous()
    srow = torch.arange(n_seq, **i32)
    cu = (torch.arange(n_seq + 1, **i32) * per).contiguous()
    past = torch.full((n_seq,), context, **i32)
    pos = torch.arange(T, **i32)
    tot = n_seq * (context + per)
    # ---- Qwen3's kernels at this width: 32 heads over 4
    h, nw, qkv = bf(T, W), bf(W), bf(T, 5120)
    gemm_case("qwen3 qkv GEMM", 5120, W, lambda w: X.gemm(h, w), 5120 * 2)
    att, xr = bf(T, 4096), bf(T, W)
    gemm_case("qwen3 o GEMM + residual", W, 4096, lambda w: X.gemm(att, w, out=xr, residual=xr), W * 4)
    add("qwen3 RMSNorm", [lambda: X.rmsnorm(h, nw, 1e-6)], T * W * 4, 0, 8)
    q, freq = bf(T, 32, D), X.inv_freq(D, 1e6, dev)
    kp, vp = bf(4, S, D), bf(4, S, D)
    add("qwen3 head norms + RoPE + KV scatter", [lambda: X.qkv_post(qkv, nw[:D], nw[:D], pos, pos, freq, q, kp, vp, 32, 4, 1e-6)], T * 5120 * 4, 0, 8)
    pairs_seen = n_seq * per * context + n_seq * per * (per + 1) // 2
    pools = [(bf(4, S, D), bf(4, S, D)) for _ in range(max(1, min(6, int(300e6 / (tot * 2048)) + 1)))]
    add("qwen3 attention", [lambda k=k, v=v: X.paged_tree_attention(q, k, v, smap, srow, cu, past, None, D ** -0.5, True, per, max_keys=context + per)
                            for k, v in pools], tot * 4 * D * 4 + T * 32 * D * 4, 4 * pairs_seen * 32 * D)
    # ---- Zasipel: a parallel layer
    head, chan = DeltaConfig(16, 8, D, D, 4), DeltaConfig(32, 32, D, D, 4, decay="channel", gate="sigmoid", decay_rank=128, gate_rank=128)
    win_cols = (16 + 2 * 4) * D
    n_act = win_cols + head.channels + 16 * D
    raw, act = torch.empty(T, 128, device=dev), torch.empty(T, n_act, dtype=torch.bfloat16, device=dev)
    gemm_case("zasipel input GEMM (both mixers)", 128 + n_act, W,
              lambda w: X.gemm_inproj(h, w, raw, 128, act, False, act=X.ACT_NONE), 512 + n_act * 2, "qwen3 qkv GEMM")
    act.copy_(bf(T, n_act))
    raw.normal_()
    lib, p = X.load(), X._p
    bias, wfreq, wq = torch.randn(win_cols, device=dev), X.pair_freq(64, 1e6, dev), bf(T, 16 * D)
    add("zasipel bias + rotation + norm + KV scatter", [lambda: X._check(lib.js_window_post(
        p(act), n_act, p(bias), 16, 4, 4, 1, D, D, D, D, D, 64, p(wfreq), 1, X.ctypes.c_float(1e-6), 0, X.ctypes.c_float(0.0), 20 * D, 1, p(pos),
        p(pos), S, T, p(wq), p(kp), p(vp),
        p(X.status_word(dev)), 0, X._stream()), "post")], T * win_cols * 4, 0, 8, "qwen3 head norms + RoPE + KV scatter")
    seen_w = n_seq * sum(min(WIN, context + i + 1) for i in range(per))
    keys_w = n_seq * min(context + per, WIN + per - 1)
    sp = X.window_attn_splits(T, 16, 4, context + per, WIN, seqs=n_seq)
    ws = {"o": torch.zeros(sp, T, 16, D, device=dev), "ml": torch.zeros(sp, T, 16, 2, device=dev)}
    wo = bf(T, 16 * D)
    add("zasipel window attention", [lambda k=k, v=v: X.window_attention_tc(wq.view(T, 16, D), k, v, smap, srow, cu, past, None, D ** -0.5, WIN, True,
                                                                           True, wo, splits=sp, ws=ws) for k, v in pools],
        keys_w * 4 * D * 4 + T * 16 * D * 4, 4 * seen_w * 16 * D, like="qwen3 attention")
    del pools
    for name, c in (("head decay", head), ("channel decay", chan)):
        C = c.channels
        pre, gate, z, b = bf(T, C) * 30, bf(T, c.heads * D), torch.randn(T, c.decays, device=dev), torch.randn(T, c.heads, device=dev)
        taps, A, dt = bf(C, c.taps), torch.linspace(-4, 0, c.heads, device=dev).to(torch.bfloat16), (bf(c.decays) - 2)
        o, on = bf(T, c.heads * D), bf(D)
        copies = max(1, min(8, int(300e6 / (n_seq * c.heads * D * D * 4)) + 1))
        st = [(torch.zeros(n_seq + 1, c.heads, D, D, device=dev), bf(n_seq + 1, c.taps, C)) for _ in range(copies)]
        io = T * (C + 2 * c.heads * D) * 2 + T * (c.decays + c.heads) * 4
        add(f"zasipel delta rule, {name} (all kernels between the GEMMs)",
            [lambda s=s: X.delta_forward(c, pre, z, b, taps, A, dt, s[0], s[1], srow, cu, past, gate, on, c.gate, 1e-6, o, max_rows=per) for s in st],
            io + n_seq * c.heads * D * D * 8, 7 * T * c.heads * D * D, like="qwen3 attention")
        del st
    low, zz, gg = bf(T, 256), torch.empty(T, 4096, device=dev), bf(T, 4096)
    gemm_case("zasipel second low-rank factors (decay fp32 | gate)", 8192, 256, lambda w: X.gemm_inproj(low, w, zz, 4096, gg, False, act=X.ACT_NONE),
              4096 * 6, "qwen3 o GEMM + residual")
    yl, yr, o2 = bf(T, W), bf(T, W), bf(T, 16 * D)
    gemm_case("zasipel output GEMM (one mixer)", W, 16 * D, lambda w: X.gemm(o2, w, out=yl), W * 2, "qwen3 o GEMM + residual")
    x32, one, hh = torch.randn(T, W, device=dev), torch.ones(W, device=dev), bf(T, W)

    def resid(**kw):
        a = dict(ya=None, bias=None, wa=None, yb=None, wb=None, ys=None, inv=None, k=0, sh=None)
        a.update(kw)
        X._check(lib.js_resid_norm(p(a["ya"]), W, p(a["bias"]), p(a["wa"]), p(a["yb"]), W, p(a["wb"]), p(a["ys"]), W, p(a["inv"]), a["k"], p(a["sh"]),
                                   W, p(one), None, X.ctypes.c_float(1e-6), p(x32), p(hh), W, None, 0, T, W, 0, X._stream()), "resid")
    add("zasipel norms of both mixers + residual", [lambda: resid(ya=yl, yb=yr, bias=one, wa=one, wb=one)], T * W * 14, 0, 8, "qwen3 RMSNorm")
    ids, tab = torch.arange(T, **i32), bf(32768, W)
    add("zasipel embedding", [lambda: X._check(lib.js_embed_f32(p(ids), p(tab), 32768, W, p(x32), p(hh), W, T, W, 0, X._stream()), "embed")],
        T * W * 8, 0, 8, "qwen3 RMSNorm")
    # ---- routed experts: 128 of 768, 8 a token
    E, k, I = 128, 8, 768
    P = T * k
    order = torch.rand(32768, E, device=dev).argsort(-1)[:, :k].to(torch.int32).contiguous()
    idx = order[:T]
    hit = int(idx.unique().numel())
    cnt = torch.bincount(idx.reshape(-1).long(), minlength=E)
    off = torch.cat((torch.zeros(1, dtype=torch.long, device=dev), cnt.cumsum(0))).to(torch.int32)
    cover = min(T, ((4 * P // E + 128 + 127) // 128) * 128)
    xs, h1, ys = bf(P, W), bf(P, I), bf(P, W)
    gu, dn = [bf(E * 2 * I, W) for _ in range(2)], [bf(E * W, I) for _ in range(3)]
    shared = "grouped gate/up + SwiGLU (the same kernel in both)", "grouped down (the same kernel in both)"
    add(shared[0], [lambda w=w: X.gemm_grouped(xs, w, h1, P, 2 * I, E, off, cover, X.EPI_SWIGLU) for w in gu],
        hit * 2 * I * W * 2 + P * (W + I) * 2, 4 * P * I * W, 4)
    add(shared[1], [lambda w=w: X.gemm_grouped(h1, w, ys, P, W, E, off, cover, X.EPI_STORE) for w in dn],
        hit * I * W * 2 + P * (W + I) * 2, 2 * P * I * W, 6)
    del gu, dn
    inv, rw = torch.randperm(P, device=dev).to(torch.int32), torch.rand(P, device=dev)
    ordr, res = torch.randperm(P, device=dev).to(torch.int32), bf(T, W)
    add("qwen3 combine + residual (invert + sum)", [lambda: X._check(lib.js_moe_combine(
        p(ys), W, p(ordr), p(rw), T, k, W, p(inv), p(res), p(res), W, 0, X._stream()), "combine")], P * W * 2 + T * W * 4, 0, 8)
    add("zasipel experts' sum + shared + norm + residual", [lambda: resid(ys=ys, inv=inv, k=k, sh=yl)], P * W * 2 + T * W * 12, 0, 8,
        "qwen3 combine + residual (invert + sum)")
    lg = torch.randn(T, E, device=dev)
    wts, ix = X.moe_route(lg, k, True)
    buf = [torch.empty(P, **i32) for _ in range(3)] + [torch.empty(E + 1, **i32), torch.empty(E, **i32)]
    if P <= 16384:
        add("qwen3 router + permutation", [lambda: (X.moe_route(lg, k, True), X._check(lib.js_moe_sort_inv(
            p(ix), p(wts), P, E, 0, E, p(buf[0]), p(rw), p(buf[3]), p(buf[4]), k, p(buf[1]), p(buf[2]), 0, X._stream()), "sort"))], T * E * 4 + P * 8, 0, 8)
        import numpy as np
        from jetspec_b200.engine.hybrid_stack import _TABLE_LAYER
        n_layers = 8
        rec = np.zeros(n_layers, dtype=_TABLE_LAYER)
        for j in range(n_layers):
            rec[j] = (order.data_ptr(), k, E, j * (2 * P + E + 1), 0)
        recs, out = torch.from_numpy(rec.view(np.uint8).reshape(-1).copy()).to(dev), torch.empty(n_layers * (2 * P + E + 1), **i32)
        add("zasipel permutations of 8 layers", [lambda: X._check(lib.js_table_sort(p(recs), n_layers, p(ids), T, 16384 // k, 32768, k, E, p(out), 0,
                                                                                    X._stream()), "sort")], n_layers * P * 12, 0, 8, "qwen3 router + permutation")
    by = {r["kernel"]: r["fraction"] for r in rows}
    for r in rows:
        if r["like"]:
            r["against_like"] = round(by[r["like"]] / max(r["fraction"], 1e-6), 2)       # > 2: more than twice as far from its roofline
    X.check_status(dev)
    return {"rows": T, "sequences": n_seq, "context": context, "peaks": note, "kernels": rows}


def main(part: str = "all", depth: int = 8) -> None:
    assert torch.cuda.is_available(), "this bench needs a GPU"
    if part in ("all", "kernels"):
        for args in ((1, 2048, 1), (16, 2048, 16), (2048, 0, 1)):
            print(json.dumps({"bench": "zasipel kernels", **kernel_table(*args)}), flush=True)
            torch.cuda.empty_cache()
    if part in ("all", "models"):
        for name, cfgs in pairs(depth).items():
            for cfg in cfgs:
                print(json.dumps({"bench": "zasipel throughput", "data": "synthetic", "dtype": "bf16", **throughput(name, cfg)}), flush=True)


if __name__ == "__main__":
    main(*sys.argv[1:2])
