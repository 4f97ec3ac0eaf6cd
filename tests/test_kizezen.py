"""Kizezen against the plain statement in ``kizezen_oracle.py``: mechanisms, whole prompts, portions, mixed batches, reuse of
pages and state slots, window edges and kept tokens, far keys and memories, long decoding, token trees and generation through
the engine's own entry points."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import kizezen_oracle as K  # noqa: E402
from kizezen_cases import (ARMS, assert_rows, band, cases, config, engine_from, latent, margin_weights, model_from, oracle_logits,  # noqa: E402
                           portions, prompt, ramp, replay, retention, rot, row_errors, window)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CASES = cases()
WEIGHTS = {k: K.random_weights(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


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


# ------------------------------------------------------------------ rotations
ROTATIONS = [rot(16, 1e4), rot(6, 500, **band(8, 1, 4, 64)), rot(64, 5e5, **band(32, 1, 4, 8192)), rot(32, 1e4, **ramp(4, 64, 8, 1)),
             rot(64, 1e4, **ramp(40, 4096, 32, 1)), rot(2, 1e4, **ramp(2, 7, 4, 2)), rot(8, 1e4, **band(1, 1, 4, 64)), rot(0, 10)]


def rotary(r, pairing):
    from jetspec_b200.models import BandScaling, RampScaling, RotaryConfig
    s = r.get("scaling")
    return RotaryConfig(r["dims"], r["base"], pairing, None if s is None else (BandScaling if "low" in s else RampScaling)(**s))


@pytest.mark.parametrize("r", ROTATIONS)
def test_frequencies_and_amplitudes(r):
    got, s = rotary(r, "half"), r.get("scaling")
    if s is None:
        want, amp = K.plain_freqs(r["dims"], r["base"]), 1.0
    elif "low" in s:
        want, amp = K.banded_freqs(r["dims"], r["base"], s), 1.0
    else:
        want, amp = K.ramped_freqs(r["dims"], r["base"], s)
    assert got.frequencies() == pytest.approx(want, rel=1e-12) and got.amplitude() == pytest.approx(amp, rel=1e-12)


def test_scalings_touch_only_some_pairs():
    plain = K.plain_freqs(64, 5e5)
    banded = rotary(ROTATIONS[2], "half").frequencies()
    kept = sum(abs(a - b) < 1e-15 for a, b in zip(plain, banded))
    divided = sum(abs(a / 32 - b) < 1e-15 for a, b in zip(plain, banded))
    assert 0 < kept < 32 and 0 < divided < 32 and kept + divided < 32        # all three bands
    ramped, plain = rotary(ROTATIONS[4], "next").frequencies(), K.plain_freqs(64, 1e4)
    share = [(a - b) / (a - a / 40) for a, b in zip(plain, ramped)]
    assert share[0] == 0 and share[-1] == pytest.approx(1) and any(0.01 < x < 0.99 for x in share)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("pairing", ["half", "next"])
@pytest.mark.parametrize("D,r", [(16, ROTATIONS[0]), (20, ROTATIONS[1]), (7, ROTATIONS[5]), (160, ROTATIONS[4]), (5, ROTATIONS[7])])
def test_rotation(arm, pairing, D, r):
    from jetspec_b200 import ops
    g = torch.Generator().manual_seed(D)
    x, pos = torch.randn(7, 3, D, generator=g).to(arm[1]), torch.tensor([0, 1, 2, 5, 63, 511, 70000])
    c = rotary(r, pairing)
    want = K.rotate(x.double(), c.frequencies(), pairing, pos, c.amplitude())
    for out in (None, torch.float32):
        got = ops.rotate(x.to(arm[0]), pos.to(arm[0]), c, out)
        assert got.dtype == (out or arm[1]) and (out is None or rel(got[:6], want[:6]) < 5e-5)
        assert rel(got[:6], want[:6]) < tol(arm, 5e-5, 1e-2) and rel(got, want) < 1e-2      # an fp32 angle at 70000: 4e-3


# ------------------------------------------------------------------ attention
def _window(arm, H, G, D, V, win, keep, scale, past, n, sink, mask=None, big=None, seed=0):
    """Product attention of ``n`` rows behind ``past`` and the formula on the same numbers."""
    from jetspec_b200 import ops
    from jetspec_b200.ops.reference import unpack_ancestor_bits
    from jetspec_b200.runtime.kv_pool import window_row_width
    dev, dt = arm
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g).to(dt)
    q, k, v = r(n, H, D), r(past + n, G, D), r(past + n, G, V)
    if big is not None:                      # one (query, key) score stands out
        k[big[1]] = 0
        k[big[1], :, 0], q[big[0], :, 0] = 6.0, 6.0
    Dp, Vp = window_row_width(D, V, dt)
    slots = torch.randperm(past + n + 40, generator=g)[:past + n].to(torch.int32)
    kp, vp = torch.zeros(G, past + n + 40, Dp, dtype=dt), torch.zeros(G, past + n + 40, Vp, dtype=dt)
    ops.window_scatter(k, v, kp, vp, slots)
    t = lambda x: x.to(dev)
    got = ops.window_attention(t(q), t(kp), t(vp), V, t(slots.view(1, -1)), i32(dev, 0), i32(dev, 0, n), i32(dev, past),
                               None if mask is None else t(mask), scale, win, t(sink) if isinstance(sink, torch.Tensor) else sink, mask is None,
                               keep_first=keep)
    anc = torch.tril(torch.ones(n, n)).bool() if mask is None else unpack_ancestor_bits(mask, n)
    pos = past + anc.sum(-1) - 1
    key_pos = torch.cat((torch.arange(past), pos))
    seen = torch.cat((torch.ones(n, past, dtype=torch.bool), anc), -1)
    seen &= (pos[:, None] - key_pos[None] < win) | (key_pos[None] < keep)
    want = torch.zeros(n, H, V, dtype=torch.float64)
    for h in range(H):
        s = q[:, h].double() @ k[:, h // (H // G)].double().T * scale
        num = sink[h].double() if isinstance(sink, torch.Tensor) else torch.zeros(()).double() if sink else None
        want[:, h] = K.softmax_with_sink(s, seen, num) @ v[:, h // (H // G)].double()
    return got.float().cpu().view(n, H, V), want


SHAPES = [(4, 2, 16, 24, 5, 3), (3, 1, 20, 8, 1, 0), (6, 3, 128, 128, 40, 66), (20, 1, 24, 16, 9, 1), (2, 1, 160, 136, 33, 4), (5, 5, 10, 12, 200, 7)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("shape", SHAPES)
def test_window_attention_with_kept_tokens_and_sinks(arm, shape):
    H, G, D, V, win, keep = shape
    sink = torch.linspace(-3.0, 4.0, H)
    for past, n, s in ((0, 7, sink), (70, 3, sink), (63, 66, sink), (17, 5, False), (130, 1, sink), (200, 20, True), (2, 3, sink)):
        got, want = _window(arm, H, G, D, V, win, keep, 1.0 / math.sqrt(D), past, n, s)
        assert rel(got, want) < tol(arm), (past, n)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("win,keep", [(1, 0), (1, 1), (2, 5), (64, 3), (65, 64), (100, 65)])
def test_window_and_kept_edges_to_the_token(arm, win, keep):
    """One key stands out; it counts as the window's last token and not one further, as the last kept token and not the next."""
    sink = torch.tensor([0.3, -1.0])
    for past, n, i in ((200, 1, 0), (150, 40, 39), (128, 5, 2), (0, 190, 189)):
        for key in {past + i - win + 1, past + i - win, keep - 1, keep}:
            if not 0 <= key <= past + i:
                continue
            got, want = _window(arm, 2, 1, 32, 32, win, keep, 0.4, past, n, sink, big=(i, key))
            assert rel(got[i], want[i]) < tol(arm), (past, key)
            if key < past + i:               # seen or not, the other answer would be far off
                seen = past + i - key < win or key < keep
                w2, k2 = (min(win, past + i - key), min(keep, key)) if seen else (win, key + 1)
                other, _ = _window(("cpu", torch.float32), 2, 1, 32, 32, w2, k2, 0.4, past, n, sink, big=(i, key))
                assert rel(other[i], want[i]) > 0.1, "the planted key does not show"


def test_sinks_take_their_share():
    """Equal scores everywhere: each head's sink takes exactly ``e^sink`` shares."""
    sink = torch.tensor([-30.0, 0.0, 2.0])
    got, want = _window(("cpu", torch.float32), 3, 3, 8, 8, 9, 0, 0.0, 20, 2, sink)
    plain, _ = _window(("cpu", torch.float32), 3, 3, 8, 8, 9, 0, 0.0, 20, 2, False)
    share = 9.0 / (9.0 + torch.exp(sink))
    assert rel(got, want) < 1e-6 and rel(got, plain.double() * share.double()[None, :, None]) < 1e-5


def _random_tree(n, g, deep):
    """Ancestor bits of a random tree, parents before children."""
    from jetspec_b200.tree.ancestor import ancestor_bits_np
    parents = [-1] + [int(torch.randint(max(0, i - deep), i, (1,), generator=g)) for i in range(1, n)]
    return parents, torch.from_numpy(ancestor_bits_np(parents, n, (n + 31) // 32).view("int32"))


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("win,keep,deep", [(200, 2, 3), (4, 6, 2), (1, 0, 3), (3, 35, 2), (20, 1, 40)])
def test_window_attention_over_token_trees(arm, win, keep, deep):
    g = torch.Generator().manual_seed(win)
    for n, past in ((7, 1), (40, 90), (70, 30)):
        _, mask = _random_tree(n, g, deep)
        got, want = _window(arm, 4, 2, 32, 24, win, keep, 0.3, past, n, torch.linspace(-1, 1, 4), mask=mask)
        assert rel(got, want) < tol(arm), (n, past)


@pytest.mark.gpu
@pytest.mark.parametrize("splits", [1, 2, 3, 12])
@pytest.mark.parametrize("H,G,win,keep", [(4, 2, 40, 3), (2, 2, 1, 70), (16, 1, 200, 0), (8, 2, 64, 64), (32, 2, 65, 129)])
def test_tensor_core_window_attention(splits, H, G, win, keep):
    """The tcgen05 kernel against the plain-core kernel: portions, decoding and trees, any number of key splits, sinks, gates."""
    from jetspec_b200.ops import cuda_ext as X
    g = torch.Generator().manual_seed(H)
    for past, n, tree in ((0, 150, False), (300, 1, False), (190, 70, False), (100, 40, True), (3, 70, True)):
        S = past + n + 30
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).cuda()
        q, kp, vp = bf(n, H, 128), bf(G, S, 128), bf(G, S, 128)
        smap = torch.randperm(S, generator=g)[:past + n].to(torch.int32).view(1, -1).cuda()
        mask = _random_tree(n, g, 5)[1].cuda() if tree else None
        sinks, gate = torch.linspace(-4, 6, H).cuda(), (2 * torch.randn(n, H + 3, generator=g)).cuda()
        args = (smap, i32("cuda", 0), i32("cuda", 0, n), i32("cuda", past), mask, 0.15, win, sinks, not tree)
        ws = {"o": torch.full((splits, n, H, 128), 7.0, device="cuda"), "ml": torch.full((splits, n, H, 2), 7.0, device="cuda")}
        out = torch.zeros(n, H * 128, dtype=torch.bfloat16, device="cuda")
        X.window_attention_tc(q, kp, vp, *args, out, splits=splits, ws=ws, keep_first=keep, gate=gate)
        want = X.window_attention(q, kp, vp, 128, *args, keep_first=keep, gate=gate)
        plain = X.window_attention(q, kp, vp, 128, *args, keep_first=keep)
        X.check_status("cuda")
        assert rel(out, want.cpu()) < 2e-2, (past, n, tree)
        gated = plain.float().view(n, H, 128) * torch.sigmoid(gate[:, :H])[..., None]
        assert rel(want, gated.view(n, -1).cpu()) < 1e-2


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("H,D,E,V,R", [(3, 12, 8, 20, 40), (2, 16, 2, 8, 8), (4, 64, 64, 64, 512), (5, 20, 0, 12, 24), (2, 30, 10, 24, 700)])
def test_latent_attention_with_a_rotated_part_and_sinks(arm, H, D, E, V, R):
    from jetspec_b200 import ops
    from jetspec_b200.runtime.kv_pool import latent_row_width
    g = torch.Generator().manual_seed(R)
    dev, dt = arm
    r = lambda *s: torch.randn(*s, generator=g).to(dt)
    for past, counts in (([0, 70], [5, 3]), ([130, 9], [1, 66])):
        S, T = 300, sum(counts)
        q, wk, wv, pool = r(T, H, D + E), r(H * D, R) * R ** -0.5, r(H * V, R) * R ** -0.5, torch.zeros(S, latent_row_width(R + E), dtype=dt)
        pool[:, : R + E] = r(S, R + E)
        smap = torch.stack([torch.randperm(S, generator=g)[:200] for _ in counts]).to(torch.int32)
        sink, cu = torch.linspace(-2, 3, H), [0, counts[0], T]
        t = lambda x: x.to(dev)
        got = ops.latent_attention(t(q), t(wk), t(wv), t(pool), t(smap), i32(dev, 0, 1), i32(dev, *cu), i32(dev, *past), None, 0.3, True, t(sink))
        for b, n in enumerate(counts):
            L = past[b] + n
            row = pool[smap[b, :L].long()].double()
            k, v = (row[:, :R] @ wk.double().T).view(L, H, D), (row[:, :R] @ wv.double().T).view(L, H, V)
            seen = torch.arange(L)[None] <= past[b] + torch.arange(n)[:, None]
            for h in range(H):
                qh = q[cu[b]:cu[b + 1], h].double()
                s = (qh[:, :D] @ k[:, h].T + qh[:, D:] @ row[:, R:R + E].T) * 0.3
                want = K.softmax_with_sink(s, seen, sink[h].double()) @ v[:, h]
                assert rel(got[cu[b]:cu[b + 1], h * V:(h + 1) * V], want) < tol(arm, 3e-5, 4e-2), (b, h)


@pytest.mark.gpu
@pytest.mark.parametrize("R,out,H", [(128, 64, 6), (320, 256, 40), (576, 512, 16), (768, 512, 3), (192, 192, 130)])
def test_tensor_core_latent_attention(R, out, H):
    """The tcgen05 kernel against the plain-core kernel: wide rows, value columns that stop before the row's end, sinks, gates."""
    from jetspec_b200.ops import cuda_ext as X
    g = torch.Generator().manual_seed(R)
    for past, counts, tree, splits in (([0, 40], [9, 1], False, 1), ([300, 65], [1, 1], False, 3), ([70], [40], True, 2)):
        T, B = sum(counts), len(counts)
        cu = [sum(counts[:i]) for i in range(B + 1)]
        qa, pool = (torch.randn(T * H, R, generator=g) * 0.4).to(torch.bfloat16).cuda(), torch.randn(500, R, generator=g).to(torch.bfloat16).cuda()
        smap = torch.stack([torch.randperm(500, generator=g)[:360] for _ in counts]).to(torch.int32).cuda()
        mask = _random_tree(T, g, 4)[1].cuda() if tree else None
        kw = dict(out_cols=out, sinks=torch.linspace(-3, 5, H).cuda(), gate=torch.randn(T, H + 1, generator=g).cuda())
        args = (qa, pool, H, smap, i32("cuda", *range(B)), i32("cuda", *cu), i32("cuda", *past), mask, 0.2, not tree, max(counts))
        want = X.latent_attention_rows(*args, impl="simt", **kw)
        ws = {"o": torch.full((splits, T * H, R), 7.0, device="cuda"), "ml": torch.full((splits, T * H, 2), 7.0, device="cuda")}
        got = X.latent_attention_rows(*args, impl="tc", splits=splits, ws=ws, **kw)
        X.check_status("cuda")
        assert rel(got[:, :out], want[:, :out].cpu()) < 2e-2, (past, counts)


@pytest.mark.parametrize("arm", ARMS)
def test_head_gate_and_exact_gelu(arm):
    from jetspec_b200 import ops
    g = torch.Generator().manual_seed(0)
    y, z = torch.randn(5, 60, generator=g).to(arm[1]), torch.randn(5, 3, generator=g) * 3
    got = ops.head_gate(y.to(arm[0]), z.to(arm[0]))
    assert rel(got, (y.double().view(5, 3, 20) * K.sigmoid(z.double())[..., None]).view(5, 60)) < tol(arm, 1e-6, 1e-2)
    x = torch.linspace(-6, 6, 400).view(4, 100).to(arm[1])
    want = K.gelu(x.double())
    assert rel(ops.gelu_erf(x.to(arm[0])), want) < tol(arm, 1e-6, 1e-2)
    tanh = torch.nn.functional.gelu(x.double(), approximate="tanh")
    assert rel(tanh, want) > 5e-5                       # in 32-bit the two gelus do not pass for each other


# ------------------------------------------------------------------ retention
def _retention_case(arm, H, D, V, counts, past, seed, dims=None):
    from jetspec_b200.models import RetentionConfig, RotaryConfig
    g = torch.Generator().manual_seed(seed)
    c = RetentionConfig(H, D, V, [1.0 - 0.5 ** (1 + i) if i else 0.2 for i in range(H)], RotaryConfig(D // 2 * 2 if dims is None else dims, 1e3))
    T, B = sum(counts), len(counts)
    r = lambda *s: torch.randn(*s, generator=g)
    q, k, v, state = r(T, H * D), r(T, H * D) * D ** -0.5, r(T, H * V).to(arm[1]), r(B + 2, H, D, V) * 0.3
    rows = torch.randperm(B + 2, generator=g)[:B].to(torch.int32)
    return c, q, k, v, state, rows, [sum(counts[:i]) for i in range(B + 1)]


def _retention_oracle(c, q, k, v, S):
    n = q.shape[0]
    q, k, v = (x.double().view(n, c.heads, -1) for x in (q, k, v))
    parts = [K.retention_rule(q[:, h], k[:, h], v[:, h], c.decay[h], S[h].double()) for h in range(c.heads)]
    return torch.stack([p[0] for p in parts], 1), torch.stack([p[1] for p in parts])


RETENTIONS = [(3, 12, 20), (2, 64, 64), (4, 128, 256), (1, 5, 3), (2, 200, 40), (3, 33, 144)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("shape", RETENTIONS)
def test_retention_over_ragged_batches(arm, shape):
    """Sequences that start (whatever their slot holds) and that continue."""
    from jetspec_b200 import ops
    counts, past = [1, 2, 19, 70, 3], [5, 0, 9, 100, 0]
    c, q, k, v, state, rows, cu = _retention_case(arm, *shape, counts, past, 1)
    t = lambda x: x.to(arm[0])
    st = t(state).clone()
    got = ops.retention(t(q), t(k), t(v), c, st, t(rows), i32(arm[0], *cu), i32(arm[0], *past), None, True)
    for i, n in enumerate(counts):
        s, r = cu[i], int(rows[i])
        want, S = _retention_oracle(c, q[s:s + n], k[s:s + n], v[s:s + n], state[r] if past[i] else torch.zeros_like(state[r]))
        assert rel(got[s:s + n], want) < 2e-5 and rel(st[r], S) < 2e-5, (i, n)
    untouched = [r for r in range(len(counts) + 2) if r not in rows.tolist()]
    assert all(torch.equal(st[r].cpu(), state[r]) for r in untouched)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("shape", RETENTIONS[:4])
def test_retention_over_token_trees(arm, shape):
    """Every node continues its parent's state; the stored state stays as it is."""
    from jetspec_b200 import ops
    n = 37
    c, q, k, v, state, rows, _ = _retention_case(arm, *shape, [n], [7], 2)
    parents, mask = _random_tree(n, torch.Generator().manual_seed(5), 6)
    t = lambda x: x.to(arm[0])
    st = t(state).clone()
    got = ops.retention(t(q), t(k), t(v), c, st, t(rows), i32(arm[0], 0, n), i32(arm[0], 7), t(mask), False)
    assert torch.equal(st.cpu(), state)
    for i in range(n):
        path = [i]
        while parents[path[0]] >= 0:
            path.insert(0, parents[path[0]])
        want, _ = _retention_oracle(c, q[path], k[path], v[path], state[int(rows[0])])
        assert rel(got[i], want[-1]) < 3e-5, i


def _fused_inputs(c, T, seed, past, counts):
    """bf16 projections of a retention layer and its rotary table; the oracle's rotated rows beside them."""
    from jetspec_b200.engine.mixers import up
    g = torch.Generator().manual_seed(seed)
    H, D, V = c.heads, c.dim, c.vdim
    cols = (up(H * D, 8), up(up(H * D, 8) + H * D, 8), up(up(up(H * D, 8) + H * D, 8) + H * V, 8))
    act = torch.randn(T, up(cols[2] + H * V, 128), generator=g).to(torch.bfloat16)
    pos = torch.cat([torch.arange(p, p + n) for p, n in zip(past, counts)])
    f = c.rot.frequencies()
    ang = pos.double()[:, None] * torch.tensor(f, dtype=torch.float64)[None]
    table = torch.zeros(T, up(len(f), 2) + 6, 2)
    table[:, 4:4 + len(f), 0], table[:, 4:4 + len(f), 1] = ang.cos(), ang.sin()
    q = K.rotate(act[:, : H * D].double().view(T, H, D), f, "half", pos).flatten(1)
    k = K.rotate(act[:, cols[0]:cols[0] + H * D].double().view(T, H, D), f, "half", pos).flatten(1) / math.sqrt(D)
    return act, cols, table, q, k, act[:, cols[1]:cols[1] + H * V], act[:, cols[2]:cols[2] + H * V]


@pytest.mark.gpu
@pytest.mark.parametrize("shape", RETENTIONS + [(2, 128, 100), (5, 64, 256), (2, 16, 1000), (1, 96, 66)])
@pytest.mark.parametrize("counts", [[1, 1, 1, 1], [1, 2, 19, 70, 3], [128, 64, 7, 300, 129], [1]])
def test_fused_retention(shape, counts):
    """The one-kernel decode step and the chunks (or the row walk, for shapes these do not take), with norm and gate."""
    from jetspec_b200.ops import cuda_ext as X
    past = [5, 0, 9, 100, 1][:len(counts)]
    c, _, _, _, state, rows, cu = _retention_case(("cuda", torch.bfloat16), *shape, counts, past, 3, dims=shape[1] // 4 * 2)
    T = sum(counts)
    act, cols, table, q, k, v, gate = _fused_inputs(c, T, 4, past, counts)
    t = lambda x: x.cuda()
    st, out = t(state).clone(), torch.zeros(T, (c.heads * c.vdim + 7) // 8 * 8, dtype=torch.bfloat16, device="cuda")
    X.retention_forward(c, t(act), cols, t(table)[:, 4:], st, t(rows), i32("cuda", *cu), i32("cuda", *past), None, 1e-5, out, max(counts))
    for i, n in enumerate(counts):
        s, r = cu[i], int(rows[i])
        want, S = _retention_oracle(c, q[s:s + n], k[s:s + n], v[s:s + n], state[r] if past[i] else torch.zeros_like(state[r]))
        assert rel(st[r], S) < 2e-5, (i, n)
        want = K.rms(want, 1e-5).reshape(n, -1) * K.silu(gate[s:s + n].double())
        assert rel(out[s:s + n, : c.heads * c.vdim], want) < 8e-3, (i, n)
    untouched = [r for r in range(len(counts) + 2) if r not in rows.tolist()]
    assert all(torch.equal(st[r].cpu(), state[r]) for r in untouched)


@pytest.mark.gpu
@pytest.mark.parametrize("shape", RETENTIONS)
def test_fused_retention_over_token_trees(shape):
    from jetspec_b200.ops import cuda_ext as X
    counts, past = [37, 150], [7, 80]
    c, _, _, _, state, rows, cu = _retention_case(("cuda", torch.bfloat16), *shape, counts, past, 6)
    trees = [_random_tree(n, torch.Generator().manual_seed(n), 5) for n in counts]
    T = sum(counts)
    act, cols, _, _, _, _, _ = _fused_inputs(c, T, 7, past, counts)
    depth = []
    for parents, _ in trees:
        d = []
        for i, p in enumerate(parents):
            d.append(0 if p < 0 else d[p] + 1)
        depth.append(d)
    pos = torch.cat([torch.tensor(d) + p for d, p in zip(depth, past)])          # rows sit at their depth
    ang = pos.double()[:, None] * torch.tensor(c.rot.frequencies(), dtype=torch.float64)[None]
    n_f = ang.shape[1]
    table = torch.zeros(T, n_f + n_f % 2, 2)
    table[:, :n_f, 0], table[:, :n_f, 1] = ang.cos(), ang.sin()
    H, D, V = c.heads, c.dim, c.vdim
    q = K.rotate(act[:, : H * D].double().view(T, H, D), c.rot.frequencies(), "half", pos).flatten(1)
    k = K.rotate(act[:, cols[0]:cols[0] + H * D].double().view(T, H, D), c.rot.frequencies(), "half", pos).flatten(1) / math.sqrt(D)
    v, gate = act[:, cols[1]:cols[1] + H * V], act[:, cols[2]:cols[2] + H * V]
    t = lambda x: x.cuda()
    W = max(m.shape[1] for _, m in trees)
    mask = torch.zeros(T, W, dtype=torch.int32)
    for (_, m), a in zip(trees, cu):
        mask[a:a + m.shape[0], : m.shape[1]] = m
    st, out = t(state).clone(), torch.zeros(T, (H * V + 7) // 8 * 8, dtype=torch.bfloat16, device="cuda")
    args = (c, t(act), cols, t(table), st, t(rows))
    X.retention_forward(*args, i32("cuda", *cu), i32("cuda", *past), t(mask), 1e-5, out, max(counts))
    assert torch.equal(st.cpu(), state)
    for b, (parents, _) in enumerate(trees):
        for i in list(range(0, counts[b], 7)) + [counts[b] - 1]:
            path = [i]
            while parents[path[0]] >= 0:
                path.insert(0, parents[path[0]])
            rows_b = [cu[b] + x for x in path]
            want, S = _retention_oracle(c, q[rows_b], k[rows_b], v[rows_b], state[int(rows[b])])
            want = K.rms(want[-1], 1e-5).reshape(-1) * K.silu(gate[cu[b] + i].double())
            assert rel(out[cu[b] + i, : H * V], want) < 8e-3, (b, i)
        st2 = t(state).clone()               # the stored state along the last node's path
        X.retention_path(c, t(act), cols, t(table), st2, i32("cuda", int(rows[b])), i32("cuda", cu[b], cu[b + 1]), i32("cuda", past[b] + len(path)),
                         i32("cuda", *path, -5), i32("cuda", len(path)))
        assert rel(st2[int(rows[b])], S) < 2e-5
    X.check_status("cuda")


# ------------------------------------------------------------------ modules and configuration
def test_mixers_alone():
    """Every mixer and feed-forward as a module, on whole sequences, against its function in the oracle."""
    from jetspec_b200.runtime import PagedAttention, PagedKVPool, build_attn_metadata
    for name in ("mixed", "ragged"):
        cfg, w = CASES[name], WEIGHTS[name]
        m = model_from(cfg, w, torch.float32, "cpu")
        pool = PagedKVPool.for_model(m.config, 4, max_seqs=2, max_seq_len=64)
        pool.reserve(1, 23)
        attn = PagedAttention(pool, build_attn_metadata(pool, [1], [0], num_query_nodes=[23]))
        h, pos = torch.randn(23, cfg["width"], generator=torch.Generator().manual_seed(1)), torch.arange(23)
        for i, L in enumerate(m.model.layers):
            spec, mix, eps = cfg["layers"][i], L.mixer, cfg["norm"]["eps"]
            with torch.no_grad():
                if spec["type"] == "attention":
                    got = mix(h, pos, lambda q, k, v: attn.window(i, mix, q, k, v))
                elif spec["type"] == "latent_attention":
                    got = mix(h, lambda q, c: attn.latent(i, mix, q, c), pos)
                else:
                    got = mix(h, pos, lambda q, k, v: attn.recur(i, mix, q, k, v))
                assert rel(got, K.MIXERS[spec["type"]](h.double(), w, f"l{i}.mix", spec["mixer"], eps)) < 2e-5, (name, i)
                if L.mlp is not None:
                    assert rel(L.mlp(h), K.feed_forward(h.double(), w, f"l{i}.mlp")) < 2e-5


def test_unknown_parts_are_refused():
    from jetspec_b200.models import KizezenConfig, family_of
    assert family_of({"architecture": "Kizezen"}).name == "kizezen"
    for change in (lambda c: c["layers"][0].update(type="something_else"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][1]["mixer"].update(heads=5), lambda c: c["layers"][0]["mixer"].update(decay=[0.5]),
                   lambda c: c["layers"][2]["mixer"].update(rot_dim=6), lambda c: c["layers"][1]["mixer"]["rot"].update(dims=40),
                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=7)):
        bad = json.loads(json.dumps(CASES["mixed"]))
        change(bad)
        with pytest.raises(ValueError):
            KizezenConfig.from_dict(bad)


def test_a_cache_layer_holds_what_its_mixer_needs():
    from jetspec_b200.models import KizezenConfig
    from jetspec_b200.runtime import PagedKVPool
    pool = PagedKVPool.for_model(KizezenConfig.from_dict(CASES["mixed"]), 4, max_seqs=2, max_seq_len=64, dtype=torch.bfloat16)
    assert [x is not None for x in pool.kv_layers] == [False, True, False, True, False, False]
    assert [x is not None for x in pool.latent_pools] == [False, False, True, False, False, True]
    assert [x is not None for x in pool.states.state] == [True, False, False, False, True, False] and not any(x is not None for x in pool.states.conv)
    assert pool.kv_layers[1][0].shape == (2, 64, 128) and pool.latent(2).shape == (64, 64) and pool.states.state[4].shape == (3, 4, 20, 12)


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", list(CASES))
def test_whole_prompt_and_residual_stream(arm, case):
    cfg, w = CASES[case], WEIGHTS[case]
    n = 150 if case == "wide" else 45
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(256, 2)
    got = replay(eng, [[("a", n)]], {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1])
    streams = []                         # the stream after every layer
    K.forward(toks[:9], w, cfg, streams=streams)
    sid, runs = eng._new_seq_id(), list(range(len(streams)))
    eng.pool.reserve(sid, 9)
    _, hid, _ = eng._forward([sid], [torch.tensor(toks[:9])], [0], taps=runs)
    for r in runs[:-1]:
        assert rel(hid[:, r * cfg["width"]:(r + 1) * cfg["width"]], streams[r]) < tol(arm, 3e-5, 3e-2), r


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case,sizes", [("mixed", [1]), ("mixed", [2]), ("mixed", [5, 2, 17]), ("one", [3]), ("one", [16, 1, 15]),
                                        ("ragged", [2, 31]), ("broad", [9, 1]), ("wide", [130, 1, 1, 2]), ("wide", [7]), ("wide", [64, 2])])
def test_portions_of_any_size_equal_the_whole(arm, case, sizes):
    """Prefill against token-by-token decoding and against portions cut inside and at the borders of pages, windows and chunks."""
    cfg, w = CASES[case], WEIGHTS[case]
    n = 150 if case == "wide" else 45
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(192, 2)
    got = replay(eng, [[("a", c)] for c in portions(n, sizes)], {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1], sizes)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "one", "ragged"])
def test_mixed_batches_equal_each_alone_and_reuse_pages_and_slots(arm, case):
    """Unequal requests, portions beside single tokens, a request that sits steps out, and a pool so small that later
    requests take the pages, slot-map rows and state slots earlier ones gave back."""
    cfg, w = CASES[case], WEIGHTS[case]
    n = {"a": 45, "b": 5, "c": 150 if case == "wide" else 18, "d": 1, "e": 45}
    req = {k: prompt(v, cfg["vocab"], seed=i if k != "e" else 0) for i, (k, v) in enumerate(n.items())}
    long_c = [("c", 149)] if case == "wide" else [("c", 17)]
    sched = ([[("a", 24), ("b", 2)], [("b", 1), ("a", 1)] + long_c, [("a", 3), ("b", 1)], [("c", 1), ("a", 2), ("b", 1), ("d", 1)]]
             + [[("a", 1), ("e", 20)], [("e", 2), ("a", 13)]] + [[("a", 1), ("e", 1)]] + [[("e", 14)], [("e", 8)]])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(48 + 16 + (160 if case == "wide" else 32) + 16, 4)
    pool = eng.pool
    for s in (*pool.states.state, *pool.latent_pools, *(x for kv in pool.kv_layers if kv is not None for x in kv)):
        if s is not None:
            s.fill_(50.0)                    # nothing may be read from a slot before its sequence wrote it
    got = replay(eng, sched, req)
    assert pool.free_page_count == pool.num_pages and not pool.resident()
    for k in req:
        assert_rows(got[k], oracle_logits(case, cfg, w, req[k]), arm[1], k)
    assert_rows(got["e"], got["a"].double(), arm[1], "reused pages")


@pytest.mark.parametrize("arm", ARMS)
def test_long_decoding(arm):
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    toks = prompt(140, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(144, 1)
    got = replay(eng, [[("a", 4)]] + [[("a", 1)]] * 136, {"a": toks})["a"]
    assert_rows(got, oracle_logits("mixed", cfg, w, toks), arm[1])


# ------------------------------------------------------------------ planted keys and far memories in the whole model
def needle_model(layer, width=64, vocab=130):
    """One layer in which a query token's heads attend almost wholly to a key token, wherever both stand: they meet in one
    unrotated coordinate that every other token's key leaves empty."""
    cfg = config(width, vocab, [(layer, 0)])
    w = K.random_weights(cfg, seed=3)
    a, b = vocab - 1, vocab - 2                 # key and query tokens
    w["embed"][:, :2] = 0.0
    w["embed"][a, 0] = w["embed"][b, 1] = 8.0
    p, m = "l0.mix", layer[1]
    if layer[0] == "attention":
        for n, c in (("q", 1), ("k", 0)):
            w[f"{p}.{n}"][m["dim"] - 1::m["dim"]] = 0.0
            w[f"{p}.{n}"][m["dim"] - 1::m["dim"], c] = 40.0
            w[f"{p}.{n}.b"][m["dim"] - 1::m["dim"]] = 0.0
        w[p + ".v"][:, 0] = 0.5
    else:
        w[p + ".dkv"][:2] = 0.0
        w[p + ".dkv"][0, 0], w[p + ".dkv"][1, 0] = 6.0, 3.0        # latent entry 0 marks the key, entry 1 its value
        w[p + ".uk"][:, 0] = 0.0
        w[p + ".uk"][0::m["dim"], 0] = 6.0
        w[p + ".uv"][:, 1] = 1.0
        hd = m["dim"] + m["rot_dim"]
        w[p + ".q"][0::hd] = 0.0
        w[p + ".q"][0::hd, 1] = 12.0
    return cfg, w, a, b


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("size,keep", [(20, 3), (64, 1), (65, 0)])
def test_keys_just_inside_and_just_outside_the_window(arm, size, keep):
    """Asked for from inside a prompt and by a decoded token, at page and tile borders, the window's edge and the kept tokens'."""
    cfg, w, a, b = needle_model(window(2, 1, 24, 16, size, keep, rot(8, 1e4, **band(4, 1, 4, 64)), scale=0.6))
    for query in (size - 1, size, size + 15, 127, 128, 150):
        for key in sorted({query - size + 1, query - size, keep - 1, keep}):
            if not 0 <= key < query:
                continue
            toks = [t % 128 for t in prompt(query + 1, 130)]
            toks[key], toks[query] = a, b
            want = K.forward(toks, w, cfg)[-1:]
            assert row_errors(K.forward(toks, w, cfg, faults={0: (query, key)})[-1:], want).max() > 0.1, "the planted key does not show"
            eng = engine_from(cfg, w, arm)
            for sizes in ([query + 1], [query, 1], [64]):
                eng.reserve_pool(160, 1)
                got = replay(eng, [[("a", c)] for c in portions(query + 1, sizes)], {"a": toks})["a"][-1:]
                assert row_errors(got, want).max() < tol(arm, 5e-5, 0.04), (key, query, sizes)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("wide", [False, True])
def test_far_keys_of_latent_attention(arm, wide):
    """One key far away among hundreds, at page and tile borders and at the first token; portions on both sides of the length
    from which keys are expanded."""
    layer = latent(2, 96, 64, 64, rot(32, 1e4, **ramp(4, 64, 8, 1))) if wide else latent(2, 12, 16, 24, rot(8, 1e4))
    cfg, w, a, b = needle_model(layer)
    eng = engine_from(cfg, w, arm)
    for query, key in ((200, 0), (200, 15), (200, 64), (255, 127), (199, 198)):
        toks = [t % 128 for t in prompt(query + 1, 130)]
        toks[key], toks[query] = a, b
        want = K.forward(toks, w, cfg)[-1:]
        assert row_errors(K.forward(toks, w, cfg, faults={0: (query, key)})[-1:], want).max() > 0.1, "the planted key does not show"
        for sizes in ([query + 1], [query, 1], [130, 2]):
            eng.reserve_pool(272, 1)
            got = replay(eng, [[("a", c)] for c in portions(query + 1, sizes)], {"a": toks})["a"][-1:]
            assert row_errors(got, want).max() < tol(arm, 5e-5, 0.04), (key, query, sizes)


@pytest.mark.parametrize("arm", ARMS)
def test_far_memories_live_in_the_state(arm):
    """A slowly forgetting head: the first token's write is read 300 tokens later, however the tokens are cut.  The oracle
    without the first tokens is far off, so a state lost on the way would show."""
    cfg = config(64, 100, [(retention(16, 16, [0.999, 1.0], rot(0, 1e4)), 0)])
    w = K.random_weights(cfg, seed=9)
    w["embed"][:, 0] = 0.0
    w["embed"][:3, 0] = 40.0                 # three tokens write strongly
    w["l0.mix.k"][:, 0] *= 32.0
    w["l0.mix.o"] *= 2.0
    toks = [0, 1, 2] + [3 + t % 97 for t in prompt(300, 100)]
    want = K.forward(toks, w, cfg)[-1:]
    assert row_errors(K.forward(toks[3:], w, cfg)[-1:], want).max() > 0.05, "the far memory does not show"
    eng = engine_from(cfg, w, arm)
    for sizes in ([303], [302, 1], [2, 64], [16, 1], [100, 3], [128, 128, 47]):
        eng.reserve_pool(304, 1)
        got = replay(eng, [[("a", c)] for c in portions(303, sizes)], {"a": toks})["a"][-1:]
        assert row_errors(got, want).max() < tol(arm, 5e-5, 0.02), sizes


@pytest.mark.parametrize("fault", ["no_sink", "no_gate"])
def test_faults_would_show(fault):
    """The random weights are such that a sink or a gate left out is far outside every tolerance used here."""
    for name in ("mixed", "wide"):
        cfg, w = CASES[name], WEIGHTS[name]
        toks = prompt(20, cfg["vocab"])
        want = oracle_logits(name, cfg, w, toks)
        for i, L in enumerate(cfg["layers"]):
            if L["type"] == "attention" or (L["type"] == "latent_attention" and fault == "no_sink"):
                assert row_errors(K.forward(toks, w, cfg, faults={i: fault}), want).max() > 0.06, (name, i)


# ------------------------------------------------------------------ token trees
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "broad"])
def test_tree_forward_commit_and_decoding_on(arm, case):
    """Every node of two trees sees its own path only; after a path is committed, decoding goes on from its state."""
    from jetspec_b200.tree import DraftTree
    cfg, w = CASES[case], WEIGHTS[case]
    pre = [prompt(19, cfg["vocab"]), prompt(8, cfg["vocab"], 1)]
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(128, 2)
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
            assert_rows(lg[r:r + 1].float().cpu(), K.forward(p + [tk[i] for i in path], w, cfg)[-1:], arm[1])
            r += 1
    chosen = [paths[0][6], paths[1][3]]
    for s, p, t, path in zip(sids, pre, trees, chosen):
        eng.pool.commit_path(s, len(p), t.num_nodes, path)
    more = [prompt(3, cfg["vocab"], 7), prompt(1, cfg["vocab"], 8)]
    lg = eng.step([(s, m, list(range(len(m)))) for s, m in zip(sids, more)])
    want = [K.forward(p + [tk[i] for i in path] + m, w, cfg)[-len(m):] for p, tk, path, m in zip(pre, toks, chosen, more)]
    assert_rows(lg.float().cpu(), torch.cat(want), arm[1])
    with pytest.raises(RuntimeError):
        eng.pool.crop(sids[0], 3)


# ------------------------------------------------------------------ generation
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "ragged"])
def test_greedy_generation_through_every_entry_point(arm, case):
    from jetspec_b200 import LLM, RandomTreeDrafter, SamplingParams
    cfg = CASES[case]
    w = WEIGHTS[case] if arm[1] == torch.float32 else margin_weights(cfg, 11)
    prompts = [prompt(n, cfg["vocab"], seed=n) for n in (5, 23, 12)]
    new = 6
    want = [K.greedy(p, w, cfg, new) for p in prompts]
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
def test_accepted_paths_of_several_nodes(arm):
    """A drafter that is often right: trees are accepted several nodes deep, so states advance along real paths."""
    from jetspec_b200 import LLM, SamplingParams
    cfg, w = CASES["mixed"], margin_weights(CASES["mixed"], 13)
    p, new = prompt(17, cfg["vocab"]), 14
    want = K.greedy(p, w, cfg, new)
    d, sp, t = _Script(p + want, cfg["vocab"]), SamplingParams(0.0, new), torch.tensor([p])
    eng = engine_from(cfg, w, arm, max_seq_len=512, max_seqs=4)
    out = eng.generate_tree(t, d, tree_depth=4, tree_width=2, budget=15, sampling_params=sp, return_stats=True)
    assert out["token_ids"] == want and max(out["accept_lengths"]) >= 3
    outs = eng.generate_tree_batch([t, t], d, block_size=5, tree_width=2, budget=15, sampling_params=sp)
    assert [o["token_ids"] for o in outs] == [want, want] and outs[0]["tpf"] > 1.5
    llm = LLM(model_from(cfg, w, arm[1], arm[0]), device=arm[0], dtype=arm[1])
    assert llm.generate_tree(t, d, block_size=5, tree_width=2, budget=15, sampling_params=sp)["token_ids"] == want
    assert llm.generate_chain(t, d, block_size=5, sampling_params=sp)["token_ids"] == want


@pytest.mark.parametrize("arm", ARMS)
def test_batch_with_a_small_pool_evicts_and_restores(arm):
    from jetspec_b200 import SamplingParams
    cfg, w = CASES["mixed"], margin_weights(CASES["mixed"], 12)
    prompts = [torch.tensor([prompt(n, cfg["vocab"], seed=n)]) for n in (30, 28, 31)]
    sp = SamplingParams(0.0, 20)
    want = [engine_from(cfg, w, arm, max_seqs=2).generate(p, sp)["token_ids"] for p in prompts]
    assert want[0] == K.greedy(prompts[0][0].tolist(), w, cfg, 20)
    for chunk in (None, 9):
        eng = engine_from(cfg, w, arm, num_pages=8, max_seq_len=64, max_seqs=4)
        assert [o["token_ids"] for o in eng.generate_batch(prompts, sp, prefill_chunk=chunk)] == want
        assert not eng.pool.resident()


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("tree", [False, True])
def test_sampling_follows_the_distribution(arm, tree):
    """How often sampled tokens fall among the oracle's 20 likeliest at a high temperature: the first token of a request, and
    the one a sampled round accepts behind a forced first token (the logit scale weighs in on both)."""
    from jetspec_b200 import RandomTreeDrafter, SamplingParams
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    p = prompt(11, cfg["vocab"])
    eng = engine_from(cfg, w, arm, max_seqs=2)
    torch.manual_seed(0)
    n, temp = 60, 4.0
    if tree:
        outs = [eng.generate_tree(torch.tensor([p]), RandomTreeDrafter(cfg["vocab"], seed=i), tree_depth=2, tree_width=2, budget=4,
                                  sampling_params=SamplingParams(temp, 2))["token_ids"] for i in range(n)]
        dists = [torch.softmax(K.forward(p + o[:1], w, cfg)[-1] / temp, -1) for o in outs]
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
    cfg = config(256, 211, [(window(4, 2, 32, 32, 19, 2, rot(16, 1e4)), 88), (retention(24, 40, [0.9, 0.98, 0.995], rot(24, 1e4)), 0),
                            (latent(4, 24, 16, 64, rot(8, 1e4, **ramp(4, 64, 8, 1))), 120)], embed=0.5, logit=0.6)
    w = margin_weights(cfg, 21)
    eng = engine_from(cfg, w, arm, max_seq_len=512, max_seqs=2)
    p = prompt(21, cfg["vocab"])
    want = K.greedy(p, w, cfg, 8)
    head = DraftHeadModel.random_init(draft_head_config(eng.cfg, 1, 5, target_layer_ids=[0, 1, 2]), seed=1, dtype=arm[1], device=arm[0])
    kw = dict(tree_depth=4, tree_width=2, budget=8)
    d, t = DraftHeadTreeDrafter(head, eng.model, block_size=5), torch.tensor([p])
    assert eng.generate_tree(t, d, target_layer_ids=head.target_layer_ids, sampling_params=SamplingParams(0.0, 8), **kw)["token_ids"] == want
    out = eng.generate_tree(t, RandomTreeDrafter(cfg["vocab"], seed=2), sampling_params=SamplingParams(1.0, 8), **kw)["token_ids"]
    assert len(out) == 8 and all(0 <= x < cfg["vocab"] for x in out)


@pytest.mark.gpu
@pytest.mark.parametrize("case", ["mixed", "wide"])
def test_long_portions(case):
    """Portions of several chunks and tiles against short ones, and the first rows against the oracle."""
    cfg, w, n = CASES[case], WEIGHTS[case], 700
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, ("cuda", torch.bfloat16))
    got = {}
    for name, sizes in (("whole", [n]), ("portions", [64, 1, 37]), ("both", [512, 1, 2])):
        eng.reserve_pool(n + 16, 1)
        got[name] = replay(eng, [[("a", c)] for c in portions(n, sizes)], {"a": toks})["a"]
    assert_rows(got["whole"], got["portions"].double(), torch.bfloat16)
    assert_rows(got["both"], got["portions"].double(), torch.bfloat16)
    assert_rows(got["whole"], oracle_logits(case, cfg, w, toks), torch.bfloat16)


# ------------------------------------------------------------------ checkpoints and the command line
def test_checkpoint_round_trip(tmp_path):
    from jetspec_b200.models import KizezenForCausalLM, load_target
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    m = model_from(cfg, w, torch.bfloat16, "cpu")
    m.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    from safetensors.torch import load_file, save_file
    t = load_file(str(tmp_path / "model.safetensors"))
    assert set(t) == set(w) and all(torch.equal(t[k].double(), w[k]) for k in w)
    m2, tok = load_target(str(tmp_path), device="cpu", dtype=torch.float32)
    assert tok is None and isinstance(m2, KizezenForCausalLM) and m2.config == m.config
    assert all(torch.equal(a.float(), b.float()) for a, b in zip(m.state_dict().values(), m2.state_dict().values()))
    other = tmp_path / "other"           # never over a file that is mapped
    m.config.save_pretrained(str(other))
    for lost in ("l1.mix.sink", "l0.mix.g", "l2.mix.dkv.norm", "l1.mix.v.b", "l2.mlp.down", "head", "embed"):
        save_file({k: v.clone() for k, v in t.items() if k != lost}, str(other / "model.safetensors"))
        with pytest.raises(KeyError):
            load_target(str(other), device="cpu", dtype=torch.float32)
    save_file({**{k: v.clone() for k, v in t.items()}, "l0.mix.sink": torch.zeros(3)}, str(other / "model.safetensors"))
    with pytest.raises(KeyError):            # a tensor the layer's mixer does not have
        load_target(str(other), device="cpu", dtype=torch.float32)


@pytest.mark.parametrize("arm", ARMS)
def test_trace_replay_command(arm, tmp_path):
    """The command: steps on standard input, logits in files, ``done`` lines, pages and slots given back at ``end``."""
    import numpy as np
    cfg, w = CASES["ragged"], WEIGHTS["ragged"]
    model, out = tmp_path / "model", tmp_path / "out"
    out.mkdir()
    model_from(cfg, w, torch.bfloat16, "cpu").save_pretrained(str(model))
    req = {k: prompt(n, cfg["vocab"], seed=n) for k, n in (("x", 40), ("y", 21), ("z", 40))}
    steps = [[("x", 20, [0, 19])], [("y", 20, []), ("x", 19, [3])], [("x", 1, [0]), ("y", 1, [0])], [("z", 39, [38, 5])], [("z", 1, [0])]]
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
