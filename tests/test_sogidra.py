"""Sogidra against the plain statement in ``sogidra_oracle.py``: mechanisms, whole prompts, portions, mixed batches, reuse of
pages and block rows, window and block edges, far keys, long decoding, token trees and generation through the engine's own entry
points."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import sogidra_oracle as S  # noqa: E402
from sogidra_cases import (ARMS, assert_rows, cases, config, diff, engine_from, margin_weights, model_from, oracle_logits, pooled,  # noqa: E402
                           portions, prompt, replay, row_errors)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CASES = cases()
WEIGHTS = {k: S.random_weights(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """Thousands of tiny products: threads only get in each other's way."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def rel(a, b):
    return ((a.double().cpu() - b.double()).abs().max() / b.double().abs().max().clamp(min=1e-9)).item()


def tol(arm, f32=2e-5, bf16=2e-2):
    return f32 if arm[1] == torch.float32 else bf16


def i32(dev, *x):
    return torch.tensor(x, dtype=torch.int32, device=dev)


# ------------------------------------------------------------------ pieces
@pytest.mark.parametrize("arm", ARMS)
def test_xielu(arm):
    from jetspec_b200 import ops
    z = torch.cat((torch.linspace(-9, 9, 395), torch.tensor([0.0, 1e-3, -1e-3, 1e-20, -60.0]))).view(4, 100).to(arm[1])
    act = torch.tensor([0.3, -1.2], dtype=torch.float64)
    want = S.xielu(z.double(), act)
    got = ops.xielu(z.to(arm[0]), float(S.softplus(act[0])), float(0.5 + S.softplus(act[1])))
    assert got.dtype == arm[1] and rel(got, want) < tol(arm, 1e-6, 1e-2)
    near = z.double().abs() < 2e-3                       # slope 1/2 at zero, from both sides
    assert rel(got.cpu()[near], want[near]) < tol(arm, 1e-5, 1e-2)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("every,coef", [(1, 0.3), (7, 0.6), (100, 1.5)])
def test_query_temperature_steps_where_it_should(arm, every, coef):
    from jetspec_b200 import ops
    pos = torch.tensor([0, 1, every - 2, every - 1, every, 2 * every - 2, 2 * every - 1, 5000]).clamp(min=0)
    x = torch.randn(len(pos), 3, 10, generator=torch.Generator().manual_seed(0)).to(arm[1])
    want = x.double() * S.temperature(pos, every, coef)[:, None, None]
    assert rel(ops.query_temperature(x.to(arm[0]), pos.to(arm[0]), every, coef), want) < tol(arm, 1e-6, 1e-2)
    assert S.temperature([every - 2], every, coef)[0] == 1.0 or every == 1
    assert S.temperature([every - 1], every, coef)[0] == pytest.approx(1.0 + coef * math.log(2.0))


@pytest.mark.parametrize("dev", ["cpu", pytest.param("cuda", marks=pytest.mark.gpu)])
@pytest.mark.parametrize("terms", [2, 5, 70])
def test_depth_average(dev, terms):
    from jetspec_b200 import ops
    g = torch.Generator().manual_seed(terms)
    x, d = [torch.randn(7, 33, generator=g) for _ in range(terms)], torch.randn(terms, generator=g).to(torch.bfloat16)
    got = ops.depth_average([t.to(dev) for t in x], d.to(dev))
    assert got.dtype == torch.float32 and rel(got, S.depth_average([t.double() for t in x], d.double())) < 1e-5


def test_norm_weights_stand_around_zero():
    from jetspec_b200.models.layers import OffsetRMSNorm
    n = OffsetRMSNorm(40, 1e-3)
    g = torch.Generator().manual_seed(0)
    x = torch.randn(5, 40, generator=g)
    assert rel(n(x), S.rms(x.double(), 1e-3)) < 1e-6
    n.weight.data = torch.randn(40, generator=g).to(torch.bfloat16)
    assert rel(n(x), S.norm(x.double(), n.weight.data.double(), 1e-3)) < 1e-6


@pytest.mark.gpu
@pytest.mark.parametrize("T,W,terms", [(1, 100, 0), (3, 96, 3), (300, 1024, 2), (5, 2304, 6), (301, 2000, 1), (320, 4096, 4), (2, 4096, 9), (9, 7000, 2),
                                       (4, 16000, 3), (2, 20000, 1)])
def test_fused_residual_step(T, W, terms):
    """Norm of the sublayer's output, sum, (at a layer's end) history and depth average, next norm, tap."""
    from jetspec_b200.ops import cuda_ext as X
    g, eps, ld = torch.Generator().manual_seed(W), 1e-3, (W + 7) // 8 * 8
    row = lambda n: torch.nn.functional.pad(torch.randn(n, W, generator=g), (0, ld - W))
    y, src, hist = row(T).to(torch.bfloat16), row(T) * 3, torch.stack([row(T) for _ in range(terms + 1)])
    w, fw, d = row(1)[0], row(1)[0], torch.randn(terms + 1, generator=g)
    c = lambda t: t.cuda()
    new = src.double() + S.rms(y.double()[:, :W], eps).new_zeros(T, ld)
    new[:, :W] += S.rms(y.double()[:, :W], eps) * w.double()[:W]
    for end in ([False] if terms == 0 else [False, True]):
        want = new if not end else S.depth_average([*hist.double()[:terms], new], d.double())
        x, h, hs = c(src).clone(), torch.full((T, ld), 7.0, dtype=torch.bfloat16, device="cuda"), c(hist).clone()
        tap = torch.zeros(T, W, dtype=torch.bfloat16, device="cuda")
        X.sandwich(c(y), x, c(w), x, c(fw), eps, h, W, **(dict(hist=hs, d=c(d)) if end else {}), tap=tap)
        assert rel(x, want) < 1e-5 and rel(tap, want[:, :W]) < 1e-2
        assert rel(h[:, :W], S.rms(want[:, :W], eps) * fw.double()[:W]) < 1e-2 and (h[:, W:] == 0).all()
        if end:
            assert rel(hs[terms], new) < 1e-6 and torch.equal(hs[:terms].cpu(), hist[:terms])


# ------------------------------------------------------------------ attention ops
def _random_tree(n, g, deep):
    """Ancestor bits of a random tree, parents before children."""
    from jetspec_b200.tree.ancestor import ancestor_bits_np
    parents = [-1] + [int(torch.randint(max(0, i - deep), i, (1,), generator=g)) for i in range(1, n)]
    return parents, torch.from_numpy(ancestor_bits_np(parents, n, (n + 31) // 32).view("int32"))


def _paths(past, n, parents):
    """Cache indices every row sees, in the order of their positions."""
    out = []
    for i in range(n):
        own = [i]
        while parents is not None and parents[own[0]] >= 0:
            own.insert(0, parents[own[0]])
        out.append(list(range(past)) + ([past + j for j in own] if parents is not None else list(range(past, past + i + 1))))
    return out


def _scattered(arm, k, v, past, n, P, maps, g, causal):
    """Pools that hold ``k``, ``v`` at shuffled slots, and the rows of the blocks whole by then at shuffled places."""
    from jetspec_b200 import ops
    from jetspec_b200.runtime.kv_pool import window_row_width
    dev, dt = arm
    L, G, Dm = k.shape
    slots = torch.randperm(L + 40, generator=g)[:L].to(torch.int32)
    Kw, Vw = window_row_width(Dm // maps, v.shape[2], dt, maps)
    kp, vp = torch.zeros(G, L + 40, Kw, dtype=dt), torch.zeros(G, L + 40, Vw, dtype=dt)
    ops.window_scatter(k, v, kp, vp, slots, maps)
    t = lambda x: x.to(dev)
    kp, vp, smap, blocks = t(kp), t(vp), t(slots.view(1, -1)), None
    if P:
        nb = L // P + 3
        kb, vb = torch.full((G, nb + 5, Kw), 90.0, dtype=dt, device=dev), torch.full((G, nb + 5, Vw), 90.0, dtype=dt, device=dev)
        bmap = t(torch.randperm(nb + 5, generator=g)[:nb].to(torch.int32).view(1, -1))
        done = past + n if causal else past
        a = done // 3                        # in two goes, as two portions would
        for p0, m in ((0, a), (a, done - a)):
            ops.pool_blocks(kp, vp, kb, vb, bmap, P, smap, i32(dev, 0), i32(dev, 0, m), i32(dev, p0))
        blocks = (kb, vb, bmap, P)
    return kp, vp, smap, blocks


def _pooled_case(arm, H, G, D, size, P, cap, scale, past, n, parents=None, mask=None, big=None, seed=0):
    """Product attention of ``n`` rows behind ``past``; the formula on the same numbers, as a function of one flipped key or block
    of one row."""
    from jetspec_b200 import ops
    dev, dt = arm
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dt)
    q, k, v = r(n, H, D), r(past + n, G, D), r(past + n, G, D)
    if big is not None:                      # one (query, key) score stands out
        k[:, :, 0] = 0
        k[big[1], :, 0], q[big[0], :, 0] = big[2], 6.0
        v[big[1]] *= 4.0
    kp, vp, smap, blocks = _scattered(arm, k, v, past, n, P, 1, g, parents is None)
    t = lambda x: x.to(dev)
    got = ops.window_attention(t(q), kp, vp, D, smap, i32(dev, 0), i32(dev, 0, n), i32(dev, past), None if mask is None else t(mask), scale, size,
                               False, mask is None, softcap=cap, blocks=blocks)
    paths = _paths(past, n, parents)

    def formula(i, flip=None):
        path = paths[i]
        pos, kk, vv = len(path) - 1, k[path].double(), v[path].double()
        near, far = (x[pos].clone() for x in S.window_and_blocks(pos + 1, size, P))
        if flip is not None:
            x = near if flip[0] == "key" else far
            x[flip[1]] = ~x[flip[1]]
        nb = far.numel()
        kb, vb = (x[: nb * P].view(nb, P, G, D).mean(1) for x in (kk, vv))
        keys, vals, seen = torch.cat((kk, kb)), torch.cat((vv, vb)), torch.cat((near, far))
        out = []
        for h in range(H):
            s = S.capped(keys[:, h // (H // G)] @ q[i, h].double() * scale, cap) if cap else keys[:, h // (H // G)] @ q[i, h].double() * scale
            out.append(S.softmax(s.masked_fill(~seen, -math.inf)) @ vals[:, h // (H // G)])
        return torch.stack(out)
    return got.float().cpu().view(n, H, D), formula


SHAPES = [(4, 2, 16, 5, 3, 8.0), (3, 1, 20, 1, 1, 30.0), (6, 2, 128, 44, 10, 45.0), (20, 1, 24, 9, 2, 3.0), (2, 1, 160, 33, 5, 20.0), (5, 5, 10, 100, 64, 0.0)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("shape", SHAPES)
def test_window_attention_with_pooled_blocks(arm, shape):
    H, G, D, size, P, cap = shape
    for past, n in ((0, 7), (70, 3), (63, 66), (17, 5), (130, 1), (200, 20), (2, 3)):
        got, formula = _pooled_case(arm, H, G, D, size, P, cap, 2.0 / math.sqrt(D), past, n)
        want = torch.stack([formula(i) for i in range(n)])
        assert rel(got, want) < tol(arm), (past, n)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("size,P", [(1, 1), (1, 4), (2, 3), (64, 2), (65, 5), (100, 16)])
def test_window_and_block_edges_to_the_token(arm, size, P):
    """One key stands out: it counts as the window's last token, not one further, and again once its whole block is behind."""
    shown = set()
    for past, n, i in ((200, 1, 0), (150, 40, 39), (128, 5, 2), (0, 190, 189), (190, 2, 1)):
        pos = past + i
        last = (pos - size + 1) // P - 1                         # last block seen
        for key in {pos - size + 1, pos - size, (last + 1) * P - 1, (last + 1) * P, last * P}:
            if not 0 <= key < pos:
                continue
            got, formula = _pooled_case(arm, 2, 1, 32, size, P, 40.0, 0.35, past, n, big=(i, key, 6.0 * min(P, 8)))
            want = formula(i)
            assert rel(got[i], want) < tol(arm, 3e-5), (past, key)
            flips = [("key", key, "window")] if key > pos - size or (key == pos - size and key // P > last) else []
            if key <= pos - size and (key // P + 1) * P <= pos + 1:          # a whole block, seen or not yet behind the window
                flips.append(("block", key // P, "seen" if key // P <= last else "not yet"))
            for what, at, kind in flips:
                assert rel(formula(i, (what, at)), want) > 0.05, ("the planted key does not show", kind)
                shown.add(kind)
    assert "seen" in shown and ("window" in shown or size == 1) and ("not yet" in shown or P == 1)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("size,P,deep", [(200, 4, 3), (4, 3, 2), (1, 1, 2), (3, 5, 1), (45, 6, 40)])
def test_pooled_blocks_over_token_trees(arm, size, P, deep):
    """Nodes see whole blocks of committed tokens and, in trees deeper than the window, of their own path."""
    g = torch.Generator().manual_seed(size)
    for n, past in ((7, 1), (40, 90), (70, 30)):
        parents, mask = _random_tree(n, g, deep)
        got, formula = _pooled_case(arm, 4, 2, 32, size, P, 20.0, 0.3, past, n, parents=parents, mask=mask)
        want = torch.stack([formula(i) for i in range(n)])
        assert rel(got, want) < tol(arm, 3e-5), (n, past)


def _diff_case(arm, H, G, D, V, scale, past, n, parents=None, mask=None, big=None, seed=0, lam=0.6, share=0.7, eps=1e-4):
    from jetspec_b200 import ops
    dev, dt = arm
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dt)
    q, k, v = r(n, H, 2, D), r(past + n, G, 2, D), r(past + n, G, V)
    if big is not None:                      # (row, key, map)
        k[:, :, :, 0] = 0
        k[big[1], :, big[2], 0], q[big[0], :, big[2], 0] = 9.0, 9.0
    kp, vp, smap, _ = _scattered(arm, k.flatten(2), v, past, n, 0, 2, g, parents is None)
    t = lambda x: x.to(dev)
    got = ops.window_attention(t(q).flatten(1, 2), kp, vp, V, smap, i32(dev, 0), i32(dev, 0, n), i32(dev, past), None if mask is None else t(mask),
                               scale, 0, False, mask is None, diff=(torch.tensor(lam, device=dev), share, eps))
    paths = _paths(past, n, parents)

    def formula(i, drop=None):
        path = [j for j in paths[i] if j != drop]
        out = []
        for h in range(H):
            a = [S.softmax(k[path, h // (H // G), m].double() @ q[i, h, m].double() * scale) @ v[path, h // (H // G)].double() for m in (0, 1)]
            out.append(share * S.rms(a[0] - lam * a[1], eps))
        return torch.stack(out)
    return got.float().cpu().view(n, H, V), formula


DIFFS = [(4, 2, 16, 24), (3, 1, 20, 8), (6, 2, 64, 128), (20, 1, 12, 16), (2, 1, 80, 136), (5, 5, 9, 11), (8, 1, 40, 88), (32, 2, 64, 100)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("shape", DIFFS)
def test_differential_attention(arm, shape):
    H, G, D, V = shape
    for past, n in ((0, 7), (70, 3), (63, 66), (130, 1), (300, 20), (2, 3)):
        got, formula = _diff_case(arm, H, G, D, V, 1.0 / math.sqrt(D), past, n)
        assert rel(got, torch.stack([formula(i) for i in range(n)])) < tol(arm, 3e-5, 2.5e-2), (past, n)
    g = torch.Generator().manual_seed(H)
    for n, past in ((7, 1), (40, 90), (70, 30)):
        parents, mask = _random_tree(n, g, 4)
        got, formula = _diff_case(arm, H, G, D, V, 1.0 / math.sqrt(D), past, n, parents=parents, mask=mask)
        assert rel(got, torch.stack([formula(i) for i in range(n)])) < tol(arm, 3e-5, 2.5e-2), (past, n, "tree")


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("which", [0, 1])
def test_far_keys_of_either_map(arm, which):
    """One key stands out in one of the maps, far back, at page and tile borders and at the first token."""
    for past, n, i in ((500, 1, 0), (400, 130, 129), (0, 260, 255)):
        for key in (0, 15, 16, 63, 64, 127, past + i - 1, past + i):
            if not 0 <= key <= past + i:
                continue
            got, formula = _diff_case(arm, 2, 1, 32, 48, 0.4, past, n, big=(i, key, which))
            want = formula(i)
            assert rel(got[i], want) < tol(arm, 3e-5), (past, key)
            assert rel(formula(i, drop=key), want) > 0.1, "the planted key does not show"


@pytest.mark.gpu
@pytest.mark.parametrize("splits", [1, 2, 3, 8, 12])
@pytest.mark.parametrize("H,G,size,P,cap", [(4, 2, 40, 3, 9.0), (2, 2, 1, 1, 0.0), (16, 1, 200, 16, 50.0), (8, 2, 64, 64, 3.0), (32, 2, 65, 5, 30.0), (4, 4, 130, 2, 0.8)])
def test_tensor_core_pooled_attention(splits, H, G, size, P, cap):
    """The tcgen05 kernel against the plain-core kernel: portions, decoding and trees, any number of key splits."""
    from jetspec_b200.ops import cuda_ext as X
    g = torch.Generator().manual_seed(H)
    for past, n, tree in ((0, 150, False), (700, 1, False), (190, 70, False), (500, 40, True), (3, 33, False)):
        if tree and size < n:
            continue
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
        q, k, v = bf(n, H, 128).cuda(), bf(past + n, G, 128), bf(past + n, G, 128)
        kp, vp, smap, blocks = _scattered(("cuda", torch.bfloat16), k, v, past, n, P, 1, g, not tree)
        mask = _random_tree(n, g, 5)[1].cuda() if tree else None
        args = (smap, i32("cuda", 0), i32("cuda", 0, n), i32("cuda", past), mask, 0.15, size, False, not tree)
        ws = {"o": torch.full((splits, n, H, 128), 7.0, device="cuda"), "ml": torch.full((splits, n, H, 2), 7.0, device="cuda")}
        out = torch.zeros(n, H * 128, dtype=torch.bfloat16, device="cuda")
        X.window_attention_tc(q, kp, vp, *args, out, splits=splits, ws=ws, softcap=cap, blocks=blocks)
        want = X.window_attention(q, kp, vp, 128, *args, softcap=cap, blocks=blocks)
        X.check_status("cuda")
        assert rel(out, want.cpu()) < 2e-2, (past, n, tree)


@pytest.mark.gpu
@pytest.mark.parametrize("splits", [1, 2, 3, 8, 12])
@pytest.mark.parametrize("H,G", [(4, 2), (2, 2), (16, 1), (8, 2), (32, 2), (3, 3)])
def test_tensor_core_differential_attention(splits, H, G):
    from jetspec_b200.ops import cuda_ext as X
    g = torch.Generator().manual_seed(H)
    d = (torch.tensor([0.55], device="cuda"), 0.65, 1e-4)
    for past, n, tree in ((0, 150, False), (700, 1, False), (190, 70, False), (100, 40, True), (3, 70, True)):
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
        q, k, v = bf(n, H, 128).cuda(), bf(past + n, G, 128), bf(past + n, G, 128)
        v[..., 100:] = 0                     # padding of narrower values
        kp, vp, smap, _ = _scattered(("cuda", torch.bfloat16), k, v, past, n, 0, 2, g, not tree)
        mask = _random_tree(n, g, 5)[1].cuda() if tree else None
        args = (smap, i32("cuda", 0), i32("cuda", 0, n), i32("cuda", past), mask, 0.15, 0, False, not tree)
        ws = {"o": torch.full((splits, n, 2 * H, 128), 7.0, device="cuda"), "ml": torch.full((splits, n, 2 * H, 2), 7.0, device="cuda")}
        out = torch.zeros(n, H * 128, dtype=torch.bfloat16, device="cuda")
        X.window_attention_tc(q, kp, vp, *args, out, splits=splits, ws=ws, diff=d, vdim=100)
        want = X.window_attention(q.view(n, 2 * H, 64), kp, vp, 100, *args, diff=d)
        X.check_status("cuda")
        assert rel(out.view(n, H, 128)[..., :100].flatten(1), want.cpu()) < 2e-2, (past, n, tree)
        assert (out.view(n, H, 128)[..., 100:] == 0).all()


# ------------------------------------------------------------------ pooled blocks in the cache
@pytest.mark.parametrize("page,P", [(16, 5), (16, 16), (16, 1), (16, 40), (8, 3), (4, 7)])
def test_every_block_has_a_row_of_its_own(page, P):
    """Rows of all blocks of all resident sequences differ, also when pages are granted one by one and used again."""
    from jetspec_b200.runtime import PagedKVPool
    pool = PagedKVPool(1, 0, 0, 40, page_size=page, max_seqs=4, max_seq_len=page * 40, kv_shapes=[(1, 4, 4)], kv_pools=[P])
    g, length = torch.Generator().manual_seed(P), {}
    for i in range(60):
        sid = int(torch.randint(0, 4, (1,), generator=g))
        grow = int(torch.randint(1, 40, (1,), generator=g))
        if sid in length and (i % 7 == 0 or not pool.allocate_slots(sid, length[sid] + grow, allow_evict=False)):
            pool.free(sid)
            del length[sid]
        elif sid not in length:
            if pool.allocate_slots(sid, grow, allow_evict=False):
                length[sid] = grow
            elif pool.has(sid):
                pool.free(sid)
        else:
            length[sid] += grow
        rows = [int(r) for s, n in length.items() for r in pool.block_maps[P][pool.state(s).row, : n // P]]
        assert len(set(rows)) == len(rows) and all(0 <= r < pool.kv_blocks[0][0].shape[1] for r in rows)


@pytest.mark.parametrize("arm", ARMS)
def test_blocks_are_means_of_what_the_cache_holds(arm):
    """Rows of ragged batches: portions that end inside, at and behind block borders, and the counted form of a committed path."""
    from jetspec_b200 import ops
    dev, dt = arm
    g, P = torch.Generator().manual_seed(4), 6
    kp, vp = torch.randn(3, 300, 10, generator=g).to(dt).to(dev), torch.randn(3, 300, 7, generator=g).to(dt).to(dev)
    smap = torch.stack([torch.randperm(300, generator=g)[:100] for _ in range(4)]).to(torch.int32).to(dev)
    bmap = torch.randperm(80, generator=g)[:64].to(torch.int32).view(4, 16).to(dev)
    counts, past, rows = [6, 1, 40, 1, 5], [0, 5, 13, 6, 24], [2, 0, 3, 1, 0]
    kb, vb = torch.full((3, 80, 10), 9.0, dtype=dt, device=dev), torch.full((3, 80, 7), 9.0, dtype=dt, device=dev)
    kb2, vb2 = kb.clone(), vb.clone()
    cu = [sum(counts[:i]) for i in range(6)]
    ops.pool_blocks(kp, vp, kb, vb, bmap, P, smap, i32(dev, *rows), i32(dev, *cu), i32(dev, *past))
    written = set()
    for n, p, r in zip(counts, past, rows):
        for b in range(p // P, (p + n) // P):
            at, slots = int(bmap[r, b]), smap[r, b * P:(b + 1) * P].long()
            written.add(at)
            assert rel(kb[:, at], kp[:, slots].double().cpu().mean(1)) < tol(arm, 1e-6, 1e-2) and rel(vb[:, at], vp[:, slots].double().cpu().mean(1)) < tol(arm, 1e-6, 1e-2)
    assert len(written) == 1 + 1 + 6 + 0 + 0 and all((kb[:, x] == 9).all() for x in range(80) if x not in written)
    if dev == "cuda":
        from jetspec_b200.ops import cuda_ext as X
        X.pool_blocks(kp, vp, kb2, vb2, bmap, P, smap, i32(dev, *rows), None, i32(dev, *[p + n for p, n in zip(past, counts)]), counts=i32(dev, *counts), most=40)
        X.check_status("cuda")
        assert torch.equal(kb, kb2) and torch.equal(vb, vb2)


# ------------------------------------------------------------------ modules and configuration
def test_mixers_alone():
    """Every mixer and feed-forward as a module, on whole sequences, against its function in the oracle."""
    from jetspec_b200.runtime import PagedAttention, PagedKVPool, build_attn_metadata
    for name in ("mixed", "ragged"):
        cfg, w = CASES[name], WEIGHTS[name]
        m = model_from(cfg, w, torch.float32, "cpu")
        pool = PagedKVPool.for_model(m.config, 4, max_seqs=2, max_seq_len=64)
        pool.reserve(1, 43)
        attn = PagedAttention(pool, build_attn_metadata(pool, [1], [0], num_query_nodes=[43]))
        h, pos, keys = torch.randn(43, cfg["width"], generator=torch.Generator().manual_seed(1)), torch.arange(43), {}
        for i, L in enumerate(m.model.layers):
            spec, mix, eps, more = cfg["layers"][i], L.mixer, cfg["norm"]["eps"], {}
            if spec["type"] == "attention":
                src = spec["mixer"].get("kv_from", i)
                if src == i:
                    keys[i] = S.differential_keys(h.double(), w, f"l{i}.mix", spec["mixer"])
                more["kv"] = keys[src]
            with torch.no_grad():
                got = mix(h, pos, lambda q, k, v: attn.window(i, mix, q, k, v))
                assert rel(got, S.MIXERS[spec["type"]](h.double(), w, f"l{i}.mix", spec["mixer"], eps, **more)) < 2e-5, (name, i)
                if L.mlp is not None:
                    assert rel(L.mlp(h), S.feed_forward(h.double(), w, f"l{i}.mlp")) < 2e-5


def test_unknown_parts_are_refused():
    from jetspec_b200.models import SogidraConfig, family_of
    assert family_of({"architecture": "Sogidra"}).name == "sogidra"
    for change in (lambda c: c["layers"][0].update(type="something_else"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][1]["mixer"].update(heads=5), lambda c: c["layers"][0]["mixer"].update(vdim=24),
                   lambda c: c["layers"][0]["mixer"]["mask"].update(pool=0), lambda c: c["layers"][3]["mixer"].update(kv_from=0),
                   lambda c: c["layers"][3]["mixer"].update(kv_from=4), lambda c: c["layers"][3]["mixer"].update(dim=10),
                   lambda c: c["layers"][5]["mixer"].update(kv_from=3)):
        bad = json.loads(json.dumps(CASES["mixed"]))
        change(bad)
        with pytest.raises(ValueError):
            SogidraConfig.from_dict(bad)


def test_a_cache_layer_holds_what_its_mixer_needs():
    from jetspec_b200.models import SogidraConfig
    from jetspec_b200.runtime import PagedKVPool
    pool = PagedKVPool.for_model(SogidraConfig.from_dict(CASES["mixed"]), 4, max_seqs=2, max_seq_len=64, dtype=torch.float32)
    assert pool.kv_layers[3] is pool.kv_layers[1] and pool.kv_layers[5] is pool.kv_layers[1] and pool.kv_layers[4] is not pool.kv_layers[1]
    assert pool.kv_layers[1][0].shape == (2, 64, 24) and pool.kv_layers[1][1].shape == (2, 64, 20)
    assert [x is not None for x in pool.kv_blocks] == [True, False, True, False, False, False, True]
    assert pool.kv_blocks[0][0].shape == (2, 16, 20) and pool.kv_blocks[6][1].shape == (1, 4, 12) and set(pool.block_maps) == {5, 3, 16}
    wide = PagedKVPool.for_model(SogidraConfig.from_dict(CASES["wide"]), 4, max_seqs=2, max_seq_len=64, dtype=torch.bfloat16)
    assert wide.kv_layers[1][0].shape == (2, 64, 128) and wide.kv_blocks[2][0].shape == (1, 4, 128)


@pytest.mark.parametrize("arm", ARMS)
def test_no_more_tokens_than_positions(arm):
    from jetspec_b200 import LLM, RandomTreeDrafter, SamplingParams
    cfg = config(64, 90, [(pooled(2, 1, 8, 4, 2), 16), (diff(2, 1, 8, 8, 0.5), 24)], positions=20)
    w = S.random_weights(cfg, seed=5)
    eng, p = engine_from(cfg, w, arm, max_seq_len=128, max_seqs=2), prompt(13, 90)
    t, d = torch.tensor([p]), RandomTreeDrafter(90, seed=1)
    if arm[1] == torch.float32:
        want = S.greedy(p, w, cfg, 8)
        assert eng.generate(t, SamplingParams(0.0, 8))["token_ids"] == want              # the last token is never fed
        assert eng.generate_tree(t, d, tree_depth=3, tree_width=2, budget=8, sampling_params=SamplingParams(0.0, 8))["token_ids"] == want
    eng.reserve_pool(128, 2)
    sp = SamplingParams(0.0, 9)
    for call in (lambda: eng.generate(t, sp), lambda: eng.generate_batch([t, t], sp), lambda: eng.generate_batch([t], sp, prefill_chunk=4),
                 lambda: eng.generate_tree(t, d, tree_depth=3, sampling_params=sp), lambda: eng.generate_tree_batch([t], d, sampling_params=sp),
                 lambda: LLM(eng.model, device=arm[0], dtype=arm[1]).generate(t, sp), lambda: eng.step([(77, list(range(21)), [])])):
        with pytest.raises(ValueError, match="positions"):
            call()


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", list(CASES))
def test_whole_prompt_and_residual_stream(arm, case):
    cfg, w = CASES[case], WEIGHTS[case]
    n = 150 if case == "wide" else 75
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(256, 2)
    got = replay(eng, [[("a", n)]], {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1])
    streams = []                         # what every layer passes on
    S.forward(toks[:39], w, cfg, streams=streams)
    sid, runs = eng._new_seq_id(), list(range(len(streams)))
    eng.pool.reserve(sid, 39)
    _, hid, _ = eng._forward([sid], [torch.tensor(toks[:39])], [0], taps=runs)
    for r in runs[:-1]:
        assert rel(hid[:, r * cfg["width"]:(r + 1) * cfg["width"]], streams[r]) < tol(arm, 3e-5, 3e-2), r


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case,sizes", [("mixed", [1]), ("mixed", [2]), ("mixed", [5, 2, 17]), ("one", [3]), ("one", [1]), ("one", [16, 1, 15]),
                                        ("ragged", [2, 31]), ("broad", [9, 1]), ("wide", [130, 1, 1, 2]), ("wide", [7]), ("wide", [64, 2])])
def test_portions_of_any_size_equal_the_whole(arm, case, sizes):
    """Prefill against token-by-token decoding and against portions cut inside and at the borders of pages, windows and blocks."""
    cfg, w = CASES[case], WEIGHTS[case]
    n = 150 if case == "wide" else 75
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(192, 2)
    got = replay(eng, [[("a", c)] for c in portions(n, sizes)], {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1], sizes)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "one", "ragged"])
def test_mixed_batches_equal_each_alone_and_reuse_pages_and_rows(arm, case):
    """Unequal requests, portions beside single tokens, a request that sits steps out, and a pool so small that later
    requests take the pages, slot-map rows and block rows earlier ones gave back."""
    cfg, w = CASES[case], WEIGHTS[case]
    n = {"a": 75, "b": 5, "c": 150 if case == "wide" else 18, "d": 1, "e": 75}
    req = {k: prompt(v, cfg["vocab"], seed=i if k != "e" else 0) for i, (k, v) in enumerate(n.items())}
    long_c = [("c", 149)] if case == "wide" else [("c", 17)]
    sched = ([[("a", 54), ("b", 2)], [("b", 1), ("a", 1)] + long_c, [("a", 3), ("b", 1)], [("c", 1), ("a", 2), ("b", 1), ("d", 1)]]
             + [[("a", 1), ("e", 20)], [("e", 2), ("a", 13)]] + [[("a", 1), ("e", 1)]] + [[("e", 44)], [("e", 8)]])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(80 + 16 + (160 if case == "wide" else 32) + 16, 4)
    pool = eng.pool
    for kv in (*pool.kv_layers, *(b for b in pool.kv_blocks if b is not None)):
        for x in kv:
            x.fill_(50.0)                    # nothing may be read from a slot before its sequence wrote it
    got = replay(eng, sched, req)
    assert pool.free_page_count == pool.num_pages and not pool.resident()
    for k in req:
        assert_rows(got[k], oracle_logits(case, cfg, w, req[k]), arm[1], k)
    assert_rows(got["e"], got["a"].double(), arm[1], "reused pages")


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "one"])
def test_long_decoding(arm, case):
    cfg, w = CASES[case], WEIGHTS[case]
    toks = prompt(170, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(176, 1)
    got = replay(eng, [[("a", 4)]] + [[("a", 1)]] * 166, {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1])


# ------------------------------------------------------------------ planted keys in the whole model
def needle_model(layer, width=64, vocab=130):
    """One layer in which a query token's heads attend almost wholly to a key token, wherever both stand: they meet in one
    coordinate that every other token's key leaves empty."""
    cfg = config(width, vocab, [(layer, 0)])
    w = S.random_weights(cfg, seed=3)
    a, b = vocab - 1, vocab - 2                 # key and query tokens
    w["embed"][:, :2] = w["pos"][:, :2] = 0.0
    w["embed"][a, 0] = w["embed"][b, 1] = 8.0
    p, m = "l0.mix", layer[1]
    per_head = m["dim"] * (2 if layer[0] == "attention" else 1)
    for n, c in (("q", 1), ("k", 0)):
        w[f"{p}.{n}"][0::per_head] = 0.0
        w[f"{p}.{n}"][0::per_head, c] = 6.0 if layer[0] == "attention" else 40.0
        if layer[0] == "attention":
            w[f"{p}.{n}.b"][0::per_head] = 0.0
    if layer[0] == "attention":
        w[p + ".v"][:, 0] = 0.5
    return cfg, w, a, b


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("size,P", [(20, 3), (64, 2), (65, 4), (1, 1)])
def test_keys_at_the_edges_of_windows_and_blocks(arm, size, P):
    """Asked for from inside a prompt and by a decoded token, at page and tile borders: the window's last token and the next one,
    tokens of the last block seen and of the next."""
    cfg, w, a, b = needle_model(pooled(2, 1, 24, size, P, cap=40.0, scale=0.7))
    shown = set()
    for query in (size - 1, size, size + 15, 127, 128, 150):
        last = (query - size + 1) // P - 1
        for key in sorted({query - size + 1, query - size, (last + 1) * P - 1, (last + 1) * P}):
            if not 0 <= key < query:
                continue
            toks = [t % 128 for t in prompt(query + 1, 130)]
            toks[key], toks[query] = a, b
            want = S.forward(toks, w, cfg)[-1:]
            if key > query - size:
                flip = ("key", query, key)
            elif (key // P + 1) * P <= query + 1:
                flip = ("block", query, key // P)
            else:
                flip = None
            if flip is not None:
                assert row_errors(S.forward(toks, w, cfg, faults={0: flip})[-1:], want).max() > 0.1, "the planted key does not show"
                shown.add((flip[0], key // P <= last))
            eng = engine_from(cfg, w, arm)
            for sizes in ([query + 1], [query, 1], [64]):
                eng.reserve_pool(160, 1)
                got = replay(eng, [[("a", c)] for c in portions(query + 1, sizes)], {"a": toks})["a"][-1:]
                assert row_errors(got, want).max() < tol(arm, 5e-5, 0.04), (key, query, sizes)
    assert ("block", True) in shown and (size == 1 or ("key", False) in shown)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("wide", [False, True])
def test_far_keys_of_differential_attention(arm, wide):
    """One key far away among hundreds, at page and tile borders and at the first token."""
    cfg, w, a, b = needle_model(diff(2, 1, 64, 128, 0.3) if wide else diff(4, 2, 12, 16, 0.5, temp=(40, 0.4)))
    eng = engine_from(cfg, w, arm)
    for query, key in ((200, 0), (200, 15), (200, 64), (255, 127), (199, 198)):
        toks = [t % 128 for t in prompt(query + 1, 130)]
        toks[key], toks[query] = a, b
        want = S.forward(toks, w, cfg)[-1:]
        assert row_errors(S.forward(toks, w, cfg, faults={0: (query, key)})[-1:], want).max() > 0.1, "the planted key does not show"
        for sizes in ([query + 1], [query, 1], [130, 2]):
            eng.reserve_pool(272, 1)
            got = replay(eng, [[("a", c)] for c in portions(query + 1, sizes)], {"a": toks})["a"][-1:]
            assert row_errors(got, want).max() < tol(arm, 5e-5, 0.04), (key, query, sizes)


@pytest.mark.parametrize("fault", ["no_temp", "no_second_map", "plain_lambda", "no_cap", "no_blocks", "normed_values", "no_average", "no_out_norm"])
def test_faults_would_show(fault):
    """The random weights are such that a mechanism left out is far outside every tolerance used here."""
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    toks = prompt(75, cfg["vocab"])
    want = oracle_logits("mixed", cfg, w, toks)
    where = {"no_temp": (1, 3, 5), "no_second_map": (1, 3, 4, 5), "plain_lambda": (1, 3, 4, 5), "no_cap": (0, 2), "no_blocks": (0, 2, 6),
             "normed_values": (0, 2, 6), "no_average": range(7), "no_out_norm": range(7)}
    for i in where[fault]:
        assert row_errors(S.forward(toks, w, cfg, faults={i: fault}), want).max() > 0.06, i


# ------------------------------------------------------------------ token trees
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "broad", "one"])
def test_tree_forward_commit_and_decoding_on(arm, case):
    """Every node of two trees sees its own path only; after a path is committed, decoding goes on over its tokens and the blocks
    it completed."""
    from jetspec_b200.tree import DraftTree
    cfg, w = CASES[case], WEIGHTS[case]
    pre = [prompt(19, cfg["vocab"]), prompt(8, cfg["vocab"], 1)]
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(192, 2)
    sids = [eng._new_seq_id() for _ in pre]
    eng.step([(s, p, []) for s, p in zip(sids, pre)])
    parents = [[-1, 0, 0, 1, 2, 3, 5, 4], [-1, 0, 1, 1]]
    toks = [[7, 8, 9, 10, 11, 12, 13, 14], [20, 21, 22, 23]]
    paths, trees = [], []
    for pa, tk, s, p in zip(parents, toks, sids, pre):
        depth = [0] * len(pa)
        for i in range(1, len(pa)):
            depth[i] = depth[pa[i]] + 1
        trees.append(DraftTree(torch.tensor(tk), torch.tensor(pa), torch.tensor(depth), len(tk)))
        eng.pool.reserve(s, len(p) + len(tk) + 4)
        of = lambda i: ([] if pa[i] < 0 else of(pa[i])) + [i]
        paths.append([of(i) for i in range(len(pa))])
    lg, _, _ = eng._forward(sids, [t.token_ids for t in trees], [len(p) for p in pre], trees=trees)
    r = 0
    for p, tk, ps in zip(pre, toks, paths):
        for path in ps:
            assert_rows(lg[r:r + 1].float().cpu(), S.forward(p + [tk[i] for i in path], w, cfg)[-1:], arm[1])
            r += 1
    chosen = [paths[0][6], paths[1][3]]
    for s, p, t, path in zip(sids, pre, trees, chosen):
        eng.pool.commit_path(s, len(p), t.num_nodes, path)
    more = [prompt(40, cfg["vocab"], 7), prompt(33, cfg["vocab"], 8)]
    lg = eng.step([(s, m, list(range(len(m)))) for s, m in zip(sids, more)])
    want = [S.forward(p + [tk[i] for i in path] + m, w, cfg)[-len(m):] for p, tk, path, m in zip(pre, toks, chosen, more)]
    assert_rows(lg.float().cpu(), torch.cat(want), arm[1])


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "ragged"])
def test_greedy_generation_through_every_entry_point(arm, case):
    from jetspec_b200 import LLM, RandomTreeDrafter, SamplingParams
    cfg = CASES[case]
    w = WEIGHTS[case] if arm[1] == torch.float32 else margin_weights(cfg, 11)
    prompts = [prompt(n, cfg["vocab"], seed=n) for n in (5, 23, 12)]
    new = 6
    want = [S.greedy(p, w, cfg, new) for p in prompts]
    t = [torch.tensor([p]) for p in prompts]
    sp = SamplingParams(0.0, new)
    eng = engine_from(cfg, w, arm, max_seq_len=512, max_seqs=8)
    assert [eng.generate(p, sp)["token_ids"] for p in t] == want
    assert [o["token_ids"] for o in eng.generate_batch(t, sp)] == want
    assert [o["token_ids"] for o in eng.generate_batch(t, sp, max_batch_size=2)] == want
    for chunk in (2, 7, 64):
        assert [o["token_ids"] for o in eng.generate_batch(t, sp, prefill_chunk=chunk)] == want
    d = RandomTreeDrafter(cfg["vocab"], seed=1)
    kw = dict(tree_depth=3, tree_width=2, budget=8, sampling_params=sp)
    assert eng.generate_tree(t[1], d, **kw)["token_ids"] == want[1]
    assert [o["token_ids"] for o in eng.generate_tree_batch(t, d, block_size=4, tree_width=2, budget=8, sampling_params=sp)] == want
    assert not eng.pool.resident()
    llm = LLM(model_from(cfg, w, arm[1], arm[0]), device=arm[0], dtype=arm[1])
    assert llm.generate(t[0], sp)["token_ids"] == want[0]
    assert llm.generate_tree(t[2], d, block_size=4, tree_width=2, budget=8, sampling_params=sp)["token_ids"] == want[2]


class _Script:
    """Drafter that proposes the true continuation (or, at every third place, something else) with a decoy beside it."""

    def __init__(self, ids, vocab):
        self.ids, self.vocab = ids, vocab

    def propose_logits(self, committed, depth, target_hidden=None):
        n = committed.shape[-1]
        out = torch.zeros(1, depth, self.vocab)
        for j in range(depth):
            tok = self.ids[min(n + j, len(self.ids) - 1)]
            out[0, j, (tok + 5) % self.vocab] = 7.0 if (n + j) % 3 == 0 else 5.0
            out[0, j, tok] = 6.0
        return out

    def propose(self, committed, k, target_hidden=None):
        n = committed.shape[-1]
        return torch.tensor([self.ids[min(n + j, len(self.ids) - 1)] if (n + j) % 3 else 0 for j in range(k)])


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "one"])
def test_accepted_paths_of_several_nodes(arm, case):
    """A drafter that is often right: trees are accepted several nodes deep, so blocks are completed by real paths."""
    from jetspec_b200 import LLM, SamplingParams
    cfg = CASES[case]
    w = WEIGHTS[case] if arm[1] == torch.float32 else margin_weights(cfg, 13)
    p, new = prompt(17, cfg["vocab"]), 30
    want = S.greedy(p, w, cfg, new)
    d, sp, t = _Script(p + want, cfg["vocab"]), SamplingParams(0.0, new), torch.tensor([p])
    eng = engine_from(cfg, w, arm, max_seq_len=512, max_seqs=4)
    out = eng.generate_tree(t, d, tree_depth=4, tree_width=2, budget=15, sampling_params=sp, return_stats=True)
    assert out["token_ids"] == want and max(out["accept_lengths"]) >= 3
    outs = eng.generate_tree_batch([t, t], d, block_size=5, tree_width=2, budget=15, sampling_params=sp)
    assert [o["token_ids"] for o in outs] == [want, want] and outs[0]["tpf"] > 1.5
    llm = LLM(model_from(cfg, w, arm[1], arm[0]), device=arm[0], dtype=arm[1])
    assert llm.generate_tree(t, d, block_size=5, tree_width=2, budget=15, sampling_params=sp)["token_ids"] == want
    assert llm.generate_chain(t, d, block_size=5, sampling_params=sp)["token_ids"] == want


@pytest.mark.gpu
def test_blocks_pooled_in_the_round_graph_equal_those_of_a_prompt():
    """After rounds that accepted real paths inside the captured graph, the block rows hold what a prompt of the same tokens
    leaves (bf16 cache, so equal up to its rounding)."""
    from jetspec_b200 import SamplingParams
    cfg = CASES["mixed"]
    w = margin_weights(cfg, 13)
    p, new = prompt(17, cfg["vocab"]), 30
    want = S.greedy(p, w, cfg, new)
    eng = engine_from(cfg, w, ("cuda", torch.bfloat16), max_seq_len=256, max_seqs=2)
    held = {}
    from jetspec_b200.runtime import PagedKVPool
    free = PagedKVPool.free

    def keep(self, sid):
        st = self._seqs.get(sid)
        if st is not None:
            for li, b in enumerate(self.kv_blocks):
                if b is not None:
                    P = self.block_sizes[li]
                    rows = self.block_maps[P][st.row, : (len(p) + new - 8) // P].long()
                    held.setdefault(li, []).append(torch.stack([x[:, rows].float().cpu() for x in b]))
        free(self, sid)
    PagedKVPool.free = keep
    try:
        out = eng.generate_tree(torch.tensor([p]), _Script(p + want, cfg["vocab"]), tree_depth=4, tree_width=2, budget=15, sampling_params=SamplingParams(0.0, new))
        eng.generate(torch.tensor([p + want]), SamplingParams(0.0, 1))
    finally:
        PagedKVPool.free = free
    assert out["token_ids"] == want and set(held) == {0, 2, 6}
    for li, (a, b) in held.items():
        assert a.shape[2] > 0 and rel(a, b) < 2e-2, li


@pytest.mark.parametrize("arm", ARMS)
def test_batch_with_a_small_pool_evicts_and_restores(arm):
    from jetspec_b200 import SamplingParams
    cfg, w = CASES["mixed"], margin_weights(CASES["mixed"], 12)
    prompts = [torch.tensor([prompt(n, cfg["vocab"], seed=n)]) for n in (30, 28, 31)]
    sp = SamplingParams(0.0, 20)
    want = [engine_from(cfg, w, arm, max_seqs=2).generate(p, sp)["token_ids"] for p in prompts]
    assert want[0] == S.greedy(prompts[0][0].tolist(), w, cfg, 20)
    for chunk in (None, 9):
        eng = engine_from(cfg, w, arm, num_pages=8, max_seq_len=64, max_seqs=4)
        assert [o["token_ids"] for o in eng.generate_batch(prompts, sp, prefill_chunk=chunk)] == want
        assert not eng.pool.resident()


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("tree", [False, True])
def test_sampling_follows_the_distribution(arm, tree):
    """How often sampled tokens fall among the oracle's 20 likeliest at a high temperature: the first token of a request, and
    the one a sampled round accepts behind a forced first token."""
    from jetspec_b200 import RandomTreeDrafter, SamplingParams
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    p = prompt(11, cfg["vocab"])
    eng = engine_from(cfg, w, arm, max_seqs=2)
    torch.manual_seed(0)
    n, temp = 60, 8.0
    if tree:
        outs = [eng.generate_tree(torch.tensor([p]), RandomTreeDrafter(cfg["vocab"], seed=i), tree_depth=2, tree_width=2, budget=4,
                                  sampling_params=SamplingParams(temp, 2))["token_ids"] for i in range(n)]
        dists = [torch.softmax(S.forward(p + o[:1], w, cfg)[-1] / temp, -1) for o in outs]
        pairs = [(d, o[1]) for d, o in zip(dists, outs)]
    else:
        probs = torch.softmax(oracle_logits("mixed", cfg, w, p)[-1] / temp, -1)
        pairs = [(probs, eng.generate(torch.tensor([p]), SamplingParams(temp, 1))["token_ids"][0]) for _ in range(n)]
    assert len({t for _, t in pairs}) > 5
    mass = sum(float(d.topk(20).values.sum()) for d, _ in pairs) / n
    hit = sum(t in d.topk(20).indices.tolist() for d, t in pairs) / n
    assert abs(hit - mass) < 4 * math.sqrt(mass * (1 - mass) / n) + 0.02


@pytest.mark.parametrize("arm", ARMS)
def test_draft_head_and_sampled_trees(arm):
    """A draft head conditioned on tapped layers (inside the round graph on the GPU) stays lossless; sampled rounds run."""
    from jetspec_b200 import DraftHeadTreeDrafter, RandomTreeDrafter, SamplingParams
    from jetspec_b200.models import DraftHeadModel, draft_head_config
    cfg = config(256, 211, [(pooled(4, 2, 32, 19, 4), 88), (diff(4, 2, 32, 40, 0.4, temp=(9, 0.3)), 0), (pooled(4, 4, 16, 40, 7), 120)])
    w = margin_weights(cfg, 21)
    eng = engine_from(cfg, w, arm, max_seq_len=512, max_seqs=2)
    p = prompt(21, cfg["vocab"])
    want = S.greedy(p, w, cfg, 8)
    head = DraftHeadModel.random_init(draft_head_config(eng.cfg, 1, 5, target_layer_ids=[0, 1, 2]), seed=1, dtype=arm[1], device=arm[0])
    kw = dict(tree_depth=4, tree_width=2, budget=8)
    d, t = DraftHeadTreeDrafter(head, eng.model, block_size=5), torch.tensor([p])
    assert eng.generate_tree(t, d, target_layer_ids=head.target_layer_ids, sampling_params=SamplingParams(0.0, 8), **kw)["token_ids"] == want
    out = eng.generate_tree(t, RandomTreeDrafter(cfg["vocab"], seed=2), sampling_params=SamplingParams(1.0, 8), **kw)["token_ids"]
    assert len(out) == 8 and all(0 <= x < cfg["vocab"] for x in out)


@pytest.mark.gpu
@pytest.mark.parametrize("case", ["mixed", "wide"])
def test_long_portions(case):
    """Portions of several tiles against short ones and against the oracle."""
    cfg, n = json.loads(json.dumps(CASES[case])), 700
    cfg["max_positions"] = n
    w = S.random_weights(cfg, seed=17)
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, ("cuda", torch.bfloat16))
    got = {}
    for name, sizes in (("whole", [n]), ("portions", [64, 1, 37]), ("both", [512, 1, 2])):
        eng.reserve_pool(n + 16, 1)
        got[name] = replay(eng, [[("a", c)] for c in portions(n, sizes)], {"a": toks})["a"]
    assert_rows(got["whole"], got["portions"].double(), torch.bfloat16)
    assert_rows(got["both"], got["portions"].double(), torch.bfloat16)
    assert_rows(got["whole"], S.forward(toks, w, cfg), torch.bfloat16)


# ------------------------------------------------------------------ checkpoints and the command line
def test_checkpoint_round_trip(tmp_path):
    from jetspec_b200.models import SogidraForCausalLM, load_target
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    m = model_from(cfg, w, torch.bfloat16, "cpu")
    m.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    from safetensors.torch import load_file, save_file
    t = load_file(str(tmp_path / "model.safetensors"))
    assert set(t) == set(w) and all(torch.equal(t[k].double(), w[k]) for k in w)
    m2, tok = load_target(str(tmp_path), device="cpu", dtype=torch.float32)
    assert tok is None and isinstance(m2, SogidraForCausalLM) and m2.config == m.config
    assert all(torch.equal(a.float(), b.float()) for a, b in zip(m.state_dict().values(), m2.state_dict().values()))
    other = tmp_path / "other"           # never over a file that is mapped
    m.config.save_pretrained(str(other))
    for lost in ("pos", "embed", "l0.norm1b", "l2.dwa", "l1.mix.lk2", "l1.mix.v.b", "l3.mix.q.b", "l0.mlp.act", "final.norm"):
        save_file({k: v.clone() for k, v in t.items() if k != lost}, str(other / "model.safetensors"))
        with pytest.raises(KeyError):
            load_target(str(other), device="cpu", dtype=torch.float32)
    for extra in ("l3.mix.k", "l0.mix.v", "l2.mlp.up"):          # a tensor the layer does not have
        save_file({**{k: v.clone() for k, v in t.items()}, extra: torch.zeros(3)}, str(other / "model.safetensors"))
        with pytest.raises(KeyError):
            load_target(str(other), device="cpu", dtype=torch.float32)


@pytest.mark.parametrize("arm", ARMS)
def test_trace_replay_command(arm, tmp_path):
    """The command: steps on standard input, logits in files, ``done`` lines, pages and rows given back at ``end``."""
    import numpy as np
    cfg, w = CASES["ragged"], WEIGHTS["ragged"]
    model, out = tmp_path / "model", tmp_path / "out"
    out.mkdir()
    model_from(cfg, w, torch.bfloat16, "cpu").save_pretrained(str(model))
    req = {k: prompt(n, cfg["vocab"], seed=n) for k, n in (("x", 60), ("y", 21), ("z", 60))}
    steps = [[("x", 40, [0, 19])], [("y", 20, []), ("x", 19, [3])], [("x", 1, [0]), ("y", 1, [0])], [("z", 59, [58, 5])], [("z", 1, [0])]]
    at, lines, want = {k: 0 for k in req}, [], []
    for i, s in enumerate(steps):
        e, end, rows = [], [], []
        for k, c, ask in s:
            e.append({"id": k, "tokens": req[k][at[k]:at[k] + c], "want": ask})
            rows += [oracle_logits("ragged", cfg, w, req[k])[at[k] + a] for a in ask]
            at[k] += c
            if at[k] == len(req[k]):
                end.append(k)
        lines.append(json.dumps({"step": i, "entries": e, "end": end}))
        want.append(torch.stack(rows) if rows else None)
    r = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", str(model), "--dtype",
                        "float32" if arm[1] == torch.float32 else "bfloat16", "--out", str(out), "--max-tokens", "128",
                        "--device", arm[0]], input="\n".join(lines) + "\n", capture_output=True, text=True, timeout=240)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    for i, rows in enumerate(want):
        path = out / f"{i}.f32"
        assert path.exists() == (rows is not None)
        if rows is not None:
            assert_rows(torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(-1, cfg["vocab"])), rows, arm[1], i)
