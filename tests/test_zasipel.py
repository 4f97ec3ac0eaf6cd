"""Zasipel against the plain statement in ``zasipel_oracle.py``: mechanisms, whole prompts, portions, mixed batches, reuse
of pages and state slots, window edges, far memories, long decoding, token trees and generation through the engine's own
entry points."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import zasipel_oracle as Z  # noqa: E402
from zasipel_cases import (ARMS, assert_rows, cases, config, delta, engine_from, margin_weights, model_from, moe, oracle_logits,  # noqa: E402
                           portions, prompt, replay, row_errors, window)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CASES = cases()
WEIGHTS = {k: Z.random_weights(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


@pytest.fixture(scope="module", autouse=True)
def one_thread():
    """Thousands of tiny products: threads only get in each other's way."""
    n = torch.get_num_threads()
    torch.set_num_threads(1)
    yield
    torch.set_num_threads(n)


def rel(a, b):
    return ((a.double().cpu() - b.double()).abs().max() / b.double().abs().max().clamp(min=1e-9)).item()


# ------------------------------------------------------------------ mechanisms alone
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("D,dims", [(16, 16), (20, 6), (7, 2), (130, 64), (8, 0)])
def test_rotation_of_neighbours_then_norm(arm, D, dims):
    from jetspec_b200 import ops
    g = torch.Generator().manual_seed(D)
    x, pos = torch.randn(9, 3, D, generator=g).to(arm[1]), torch.tensor([0, 1, 2, 5, 63, 64, 511, 4000, 70000])
    want = Z.rotate(x.double(), dims, 3e4, pos)
    got = ops.rotate_norm(x.to(arm[0]), pos.to(arm[0]), dims, 3e4, None)
    tol = 1e-2 if arm[1] == torch.bfloat16 else 5e-3      # fp32 angles: an ulp at position 70000 is 4e-3
    assert rel(got, want) < tol
    assert rel(got[:6], want[:6]) < (1e-2 if arm[1] == torch.bfloat16 else 3e-5)
    got = ops.rotate_norm(x.to(arm[0]) * 1e-3, pos.to(arm[0]), dims, 3e4, 1e-6)      # eps weighs in, inside the root
    assert rel(got[:6], Z.rms(Z.rotate((x * 1e-3).double(), dims, 3e4, pos), 1e-6)[:6]) < (1e-2 if arm[1] == torch.bfloat16 else 3e-5)


def _attention(arm, H, G, D, V, win, scale, past, n, sink=True, mask=None, big=None, seed=0):
    """Product attention of ``n`` rows behind ``past`` and the oracle's formula on the same numbers."""
    from jetspec_b200 import ops
    from jetspec_b200.runtime.kv_pool import window_row_width
    from jetspec_b200.ops.reference import unpack_ancestor_bits
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
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device=dev)
    got = ops.window_attention(t(q), t(kp), t(vp), V, t(slots.view(1, -1)), i32(0), i32(0, n), i32(past), None if mask is None else t(mask),
                               scale, win, sink, mask is None)
    anc = torch.tril(torch.ones(n, n)).bool() if mask is None else unpack_ancestor_bits(mask, n)
    pos = past + anc.sum(-1) - 1
    want = torch.zeros(n, H, V, dtype=torch.float64)
    for i in range(n):
        js = [j for j in range(past) if int(pos[i]) - j < win] + [past + j for j in range(n) if anc[i, j] and int(pos[i] - pos[j]) < win]
        for h in range(H):
            s = (k[js, h // (H // G)].double() @ q[i, h].double()) * scale
            top = max(float(s.max()), 0.0)
            e = torch.exp(s - top)
            want[i, h] = (e / ((math.exp(-top) if sink else 0.0) + e.sum())) @ v[js, h // (H // G)].double()
    return got.float().cpu().view(n, H, V), want


SHAPES = [(4, 2, 16, 24, 5), (3, 1, 20, 8, 1), (6, 3, 128, 128, 40), (20, 1, 24, 16, 9), (2, 1, 160, 136, 33), (5, 5, 10, 12, 200)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("shape", SHAPES)
def test_window_attention_with_and_without_a_sink(arm, shape):
    H, G, D, V, win = shape
    for past, n, sink in ((0, 7, True), (70, 3, True), (63, 66, True), (17, 5, False), (130, 1, True)):
        got, want = _attention(arm, H, G, D, V, win, 1.0 / math.sqrt(D), past, n, sink)
        assert rel(got, want) < (2e-5 if arm[1] == torch.float32 else 2e-2), (past, n, sink)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("win", [1, 2, 64, 65, 100])
def test_window_edge_to_the_token(arm, win):
    """One key stands out; it counts as the window's last token and not one token further, in portions and decoded."""
    for past, n, i in ((150, 1, 0), (100, 40, 39), (128, 5, 2), (0, 140, 139)):
        for far in (win - 1, win):
            key = past + i - far
            if key < 0:
                continue
            got, want = _attention(arm, 2, 1, 32, 32, win, 0.4, past, n, big=(i, key))
            assert rel(got[i], want[i]) < (2e-5 if arm[1] == torch.float32 else 2e-2)
            other, _ = _attention(("cpu", torch.float32), 2, 1, 32, 32, win + (1 if far == win else -1), 0.4, past, n, big=(i, key)) \
                if far == win or win > 1 else (want + 1, None)
            assert rel(other[i], want[i]) > 0.2, "the planted key does not show"


def test_sink_takes_its_share():
    """All scores far below 0: nearly all weight falls on the sink, and without it the output is a plain mean."""
    with_sink, want = _attention(("cpu", torch.float32), 1, 1, 8, 8, 9, 1e-4, 20, 2)
    assert rel(with_sink, want) < 1e-5
    without, _ = _attention(("cpu", torch.float32), 1, 1, 8, 8, 9, 1e-4, 20, 2, sink=False)
    assert rel(without, want * 10 / 9) < 1e-3


def _random_tree(n, g, deep):
    """Ancestor bits of a random tree, parents before children."""
    from jetspec_b200.tree.ancestor import ancestor_bits_np
    parents = [-1] + [int(torch.randint(max(0, i - deep), i, (1,), generator=g)) for i in range(1, n)]
    return parents, torch.from_numpy(ancestor_bits_np(parents, n, (n + 31) // 32).view("int32"))


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("win,deep", [(200, 3), (4, 2), (1, 3), (20, 40)])
def test_window_attention_over_token_trees(arm, win, deep):
    g = torch.Generator().manual_seed(win)
    for n, past in ((7, 0), (40, 90), (70, 30)):
        _, mask = _random_tree(n, g, deep)
        got, want = _attention(arm, 4, 2, 32, 24, win, 0.3, past, n, mask=mask)
        assert rel(got, want) < (2e-5 if arm[1] == torch.float32 else 2e-2), (n, past)


def _delta_case(cfg, decay, arm, counts, past, seed, mask=None):
    """Inputs of one ragged ``delta_mix`` call and the oracle's per-sequence results."""
    from jetspec_b200.models import DeltaConfig
    dev, dt = arm
    c = DeltaConfig(*cfg, decay=decay)
    g = torch.Generator().manual_seed(seed)
    r = lambda *s: torch.randn(*s, generator=g)
    B, T = len(counts), sum(counts)
    pre, z, b = r(T, c.channels).to(dt), r(T, c.decays), r(T, c.heads)
    taps, A_log, dt_bias = (r(c.channels, c.taps) * 0.6).to(dt), torch.linspace(-4.0, 2.0, c.heads).to(dt), (r(c.decays) - 1).to(dt)
    state, conv = r(B + 2, c.heads, c.dim, c.vdim) * 0.3, r(B + 2, c.taps, c.channels).to(dt)
    rows = torch.randperm(B + 2, generator=g)[:B].to(torch.int32)
    return c, pre, z, b, taps, A_log, dt_bias, state, conv, rows


def _stored_rows(ring, past):
    """The ``taps - 1`` rows before position ``past``, oldest first, zeros before the start."""
    n = ring.shape[0]
    return torch.stack([ring[(past - m) % n] if past >= m else torch.zeros_like(ring[0]) for m in range(n - 1, 0, -1)]
                       + [ring[0]])[: n - 1]


def _delta_oracle(c, y, z, b, taps, A_log, dt_bias, S):
    """Read-outs and final state of one chain; ``y`` holds ``taps - 1`` stored rows in front."""
    y, taps, S = y.double(), taps.double(), S.double().clone()
    n, H, G, D, V = z.shape[0], c.heads, c.kv_heads, c.dim, c.vdim
    conv = torch.stack([Z.silu(sum(taps[:, j] * y[t + j] for j in range(c.taps))) for t in range(n)])
    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q = unit(conv[:, :G * D].view(n, G, D)) / math.sqrt(D)
    k = unit(conv[:, G * D:2 * G * D].view(n, G, D))
    v = conv[:, 2 * G * D:].view(n, H, V)
    gl = -torch.exp(A_log.double())[:, None] * Z.softplus(z.double() + dt_bias.double()).view(n, H, -1)
    out = torch.zeros(n, H, V, dtype=torch.float64)
    for t in range(n):
        for h in range(H):
            kh, qh = k[t, h // (H // G)], q[t, h // (H // G)]
            S[h] *= torch.exp(gl[t, h])[:, None]
            u = torch.sigmoid(b[t, h].double()) * (v[t, h] - S[h].T @ kh)
            S[h] += torch.outer(kh, u)
            out[t, h] = S[h].T @ qh
    return out, S


DELTAS = [(3, 1, 12, 20, 4), (2, 2, 64, 64, 3), (4, 2, 128, 96, 5), (1, 1, 5, 3, 1), (2, 1, 200, 40, 2), (2, 1, 32, 144, 17)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("decay", ["head", "channel"])
@pytest.mark.parametrize("cfg", DELTAS)
def test_delta_rule_over_ragged_batches(arm, decay, cfg):
    """Sequences that start (whatever their slot holds) and that continue, portions shorter and longer than the taps."""
    from jetspec_b200 import ops
    counts, past = [1, 2, 19, 70, 3], [5, 0, 9, 100, 0]
    c, pre, z, b, taps, A_log, dt_bias, state, conv, rows = _delta_case(cfg, decay, arm, counts, past, 1)
    dev = arm[0]
    t = lambda x: x.to(dev)
    st, cv = t(state).clone(), t(conv).clone()
    cu = [sum(counts[:i]) for i in range(len(counts) + 1)]
    got = ops.delta_mix(t(pre), t(z), t(b), t(taps), t(A_log), t(dt_bias), c, st, cv, t(rows), t(torch.tensor(cu, dtype=torch.int32)),
                        t(torch.tensor(past, dtype=torch.int32)), None, True)
    for i, n in enumerate(counts):
        s, r = cu[i], int(rows[i])
        S0 = state[r] if past[i] else torch.zeros_like(state[r])
        y = torch.cat((_stored_rows(conv[r], past[i]), pre[s:s + n]))
        want, S = _delta_oracle(c, y, z[s:s + n], b[s:s + n], taps, A_log, dt_bias, S0)
        assert rel(got[s:s + n], want) < 2e-5, (i, n)
        assert rel(st[r], S) < 2e-5, (i, n)
        if c.taps > 1:                   # what the next token will read
            assert torch.equal(_stored_rows(cv[r].cpu(), past[i] + n), y[-(c.taps - 1):])
    untouched = [r for r in range(len(counts) + 2) if r not in rows.tolist()]
    assert all(torch.equal(st[r].cpu(), state[r]) for r in untouched)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("decay", ["head", "channel"])
@pytest.mark.parametrize("cfg", DELTAS[:3])
def test_delta_rule_over_token_trees(arm, decay, cfg):
    """Every node continues its parent's state; the stored state and convolution inputs stay as they are."""
    from jetspec_b200 import ops
    n = 37
    c, pre, z, b, taps, A_log, dt_bias, state, conv, rows = _delta_case(cfg, decay, arm, [n], [7], 2)
    parents, mask = _random_tree(n, torch.Generator().manual_seed(5), 6)
    dev = arm[0]
    t = lambda x: x.to(dev)
    i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device=dev)
    st, cv = t(state).clone(), t(conv).clone()
    got = ops.delta_mix(t(pre), t(z), t(b), t(taps), t(A_log), t(dt_bias), c, st, cv, t(rows), i32(0, n), i32(7), t(mask), False)
    assert torch.equal(st.cpu(), state) and torch.equal(cv.cpu(), conv)
    r = int(rows[0])
    for i in range(n):
        path = [i]
        while parents[path[0]] >= 0:
            path.insert(0, parents[path[0]])
        want, _ = _delta_oracle(c, torch.cat((_stored_rows(conv[r], 7), pre[path])), z[path], b[path], taps, A_log, dt_bias, state[r])
        assert rel(got[i], want[-1]) < 3e-5, i


@pytest.mark.gpu
@pytest.mark.parametrize("decay", ["head", "channel"])
@pytest.mark.parametrize("cfg", DELTAS + [(2, 1, 128, 256, 4), (4, 4, 64, 128, 2), (1, 1, 100, 12, 3), (3, 1, 16, 8, 4)])
@pytest.mark.parametrize("counts", [[1, 1, 1, 1], [1, 2, 19, 70, 3], [8, 16, 7, 64, 9]])
def test_fused_delta_forms(decay, cfg, counts):
    """The one-kernel decode step and the blocks of 8 rows (where the shape takes them) with norm and gate; decays from
    none to forgetting everything within a token."""
    from jetspec_b200.ops import cuda_ext as X
    arm = ("cuda", torch.bfloat16)
    past = [5, 0, 9, 100, 1][:len(counts)]
    c, pre, z, b, taps, A_log, dt_bias, state, conv, rows = _delta_case(cfg, decay, arm, counts, past, 3)
    A_log = torch.linspace(-6.0, 4.0, c.heads).to(torch.bfloat16)
    g = torch.Generator().manual_seed(4)
    T = sum(counts)
    gate, norm = torch.randn(T, c.heads * c.vdim, generator=g).to(torch.bfloat16), torch.randn(c.vdim, generator=g).to(torch.bfloat16)
    t = lambda x: x.cuda()
    st, cv = t(state).clone(), t(conv).clone()
    out = torch.zeros(T, c.heads * c.vdim, dtype=torch.bfloat16, device="cuda")
    cu = [sum(counts[:i]) for i in range(len(counts) + 1)]
    n = X.delta_forward(c, t(pre), t(z), t(b), t(taps), t(A_log), t(dt_bias), st, cv, t(rows), t(torch.tensor(cu, dtype=torch.int32)),
                        t(torch.tensor(past, dtype=torch.int32)), t(gate), t(norm), "sigmoid", 1e-6, out, max(counts))
    assert n == (1 if max(counts) == 1 and X.delta_step_ok(c) else 3)
    for i, m in enumerate(counts):
        s, r = cu[i], int(rows[i])
        y = torch.cat((_stored_rows(conv[r], past[i]), pre[s:s + m]))
        want, S = _delta_oracle(c, y, z[s:s + m], b[s:s + m], taps, A_log, dt_bias, state[r] if past[i] else torch.zeros_like(state[r]))
        assert rel(st[r], S) < 2e-5, (i, m)
        want = (Z.rms(want, 1e-6) * norm.double()).reshape(m, -1) * Z.sigmoid(gate[s:s + m].double())
        assert rel(out[s:s + m], want) < 6e-3, (i, m)
        if c.taps > 1:
            assert torch.equal(_stored_rows(cv[r].cpu(), past[i] + m), y[-(c.taps - 1):])


@pytest.mark.gpu
@pytest.mark.parametrize("splits", [1, 2, 3, 12])
@pytest.mark.parametrize("H,G,win,sink", [(4, 2, 40, True), (2, 2, 1, True), (16, 1, 200, False), (8, 2, 64, True), (32, 2, 65, True)])
def test_tensor_core_window_attention(splits, H, G, win, sink):
    """The tcgen05 kernel against the plain-core kernel: portions, decoding and trees, any number of key splits."""
    from jetspec_b200.ops import cuda_ext as X
    g = torch.Generator().manual_seed(H)
    for past, n, tree in ((0, 150, False), (300, 1, False), (190, 70, False), (100, 40, True), (3, 70, True)):
        S = past + n + 30
        bf = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16).cuda()
        q, kp, vp = bf(n, H, 128), bf(G, S, 128), bf(G, S, 128)
        smap = torch.randperm(S, generator=g)[:past + n].to(torch.int32).view(1, -1).cuda()
        i32 = lambda *x: torch.tensor(x, dtype=torch.int32, device="cuda")
        mask = _random_tree(n, g, 5)[1].cuda() if tree else None
        args = (smap, i32(0), i32(0, n), i32(past), mask, 0.15, win, sink, not tree)
        ws = {"o": torch.full((splits, n, H, 128), 7.0, device="cuda"), "ml": torch.full((splits, n, H, 2), 7.0, device="cuda")}
        out = torch.zeros(n, H * 128, dtype=torch.bfloat16, device="cuda")
        X.window_attention_tc(q, kp, vp, *args, out, splits=splits, ws=ws)
        want = X.window_attention(q, kp, vp, 128, *args)
        X.check_status("cuda")
        assert rel(out, want.cpu()) < 2e-2, (past, n, tree)


@pytest.mark.parametrize("kind", ["silu", "sigmoid"])
@pytest.mark.parametrize("arm", ARMS)
def test_gated_head_norm(arm, kind):
    from jetspec_b200 import ops
    g = torch.Generator().manual_seed(0)
    o, w, gate = torch.randn(5, 3, 20, generator=g) * 1e-3, torch.randn(20, generator=g).to(arm[1]), torch.randn(5, 60, generator=g).to(arm[1])
    act = Z.silu if kind == "silu" else Z.sigmoid
    want = (Z.rms(o.double(), 1e-6) * w.double()).reshape(5, 60) * act(gate.double())
    got = ops.gated_head_norm(o.to(arm[0]), w.to(arm[0]), gate.to(arm[0]), kind, 1e-6)
    assert rel(got, want) < (1e-5 if arm[1] == torch.float32 else 1e-2)


def test_blocks_alone():
    """Both mixers and the experts as modules, on whole sequences, against their functions in the oracle."""
    from jetspec_b200.runtime import PagedAttention, PagedKVPool, build_attn_metadata
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    m = model_from(cfg, w, torch.float32, "cpu")
    pool = PagedKVPool.for_model(m.config, 4, max_seqs=2, max_seq_len=64)
    pool.reserve(1, 23)
    attn = PagedAttention(pool, build_attn_metadata(pool, [1], [0], num_query_nodes=[23]))
    toks = prompt(23, cfg["vocab"])
    h = torch.randn(23, cfg["width"], generator=torch.Generator().manual_seed(1))
    pos = torch.arange(23)
    for i, L in enumerate(m.model.layers):
        p, spec, eps = f"l{i}", cfg["layers"][i], cfg["norm"]["eps"]
        recur = lambda pre, z, b: attn.delta(i, L.delta, pre, z, b)
        with torch.no_grad():
            if spec["type"] == "parallel":
                got = L.mixer(h, pos, lambda q, k, v: attn.window(i, L.mixer.left, q, k, v), recur)
                assert rel(got, Z.parallel(h.double(), w, p + ".mix", spec["mixer"], eps)) < 2e-5
            else:
                assert rel(L.mixer(h, recur), Z.channel_delta(h.double(), w, p + ".mix", spec["mixer"], eps)) < 2e-5
            if L.mlp is not None:
                assert rel(L.mlp(h, torch.tensor(toks)), Z.table_moe(h.double(), w, p + ".mlp", spec["mlp"], toks)) < 2e-5


def test_unknown_parts_are_refused(tmp_path):
    from jetspec_b200.models import ZasipelConfig, ZasipelForCausalLM, family_of
    assert family_of({"architecture": "Zasipel"}).name == "zasipel"
    for change in (lambda c: c["layers"][0].update(type="something_else"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                   lambda c: c["layers"][0]["mixer"]["left"].update(heads=5)):
        bad = json.loads(json.dumps(CASES["mixed"]))
        change(bad)
        with pytest.raises(ValueError):
            ZasipelConfig.from_dict(bad)
    m = model_from(CASES["mixed"], WEIGHTS["mixed"], torch.bfloat16, "cpu")
    m.model.layers[0].mlp.table[3, 0] = 7
    m.save_pretrained(str(tmp_path))
    with pytest.raises(ValueError):
        ZasipelForCausalLM.from_pretrained(str(tmp_path))


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
    Z.forward(toks[:9], w, cfg, streams=streams)
    sid, runs = eng._new_seq_id(), list(range(len(streams)))
    eng.pool.reserve(sid, 9)
    _, hid, _ = eng._forward([sid], [torch.tensor(toks[:9])], [0], taps=runs)
    for r in runs[:-1]:
        assert rel(hid[:, r * cfg["width"]:(r + 1) * cfg["width"]], streams[r]) < (3e-5 if arm[1] == torch.float32 else 3e-2), r


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case,sizes", [("mixed", [1]), ("mixed", [2]), ("mixed", [5, 2, 17]), ("one", [3]), ("one", [16, 1, 15]),
                                        ("ragged", [2, 31]), ("broad", [9, 1]), ("wide", [130, 1, 1, 2]), ("wide", [7]), ("wide", [64, 2])])
def test_portions_of_any_size_equal_the_whole(arm, case, sizes):
    """Prefill against token-by-token decoding and against portions cut inside and at the borders of pages and windows."""
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
    for s in (*eng.pool.states.state, *eng.pool.states.conv):
        s.fill_(50.0)                    # nothing may be read from a slot before its sequence wrote it
    got = replay(eng, sched, req)
    assert eng.pool.free_page_count == eng.pool.num_pages and not eng.pool.resident()
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


# ------------------------------------------------------------------ window edges and far memories in the whole model
def needle_model(size, width=64, vocab=130):
    """One parallel layer in which a query token's head attends almost wholly to a key token inside its window: they meet
    in one unrotated coordinate that every other token's key leaves empty."""
    m = window(2, 1, 24, 16, size, 8, scale=0.6)
    cfg = config(width, vocab, [(m, delta(1, 1, 8, 8, 2), None)])
    w = Z.random_weights(cfg, seed=3)
    a, b = vocab - 1, vocab - 2                 # key and query tokens
    w["embed"][:, :2] = 0.0
    w["embed"][a, 0] = w["embed"][b, 1] = 8.0
    p = "l0.mix.left"
    for n, c in (("q", 1), ("k", 0)):
        w[f"{p}.{n}"][23] = 0.0
        w[f"{p}.{n}"][23, c] = 16.0
        w[f"{p}.{n}.b"][23] = 0.0
    w["l0.mix.left.v"][:, 0] = 0.5
    return cfg, w, a, b


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("size", [20, 64, 65])
def test_keys_just_inside_and_just_outside_the_window(arm, size):
    """Asked for from inside a prompt and by a decoded token, at page and tile borders and from the first tokens on."""
    cfg, w, a, b = needle_model(size)
    wider = json.loads(json.dumps(cfg))
    for query in (size - 1, size, size + 15, 127, 128, 150):
        for key in (query - size + 1, query - size):
            if key < 0:
                continue
            toks = [t % 128 for t in prompt(query + 1, 130)]
            toks[key], toks[query] = a, b
            want = Z.forward(toks, w, cfg)[-1:]
            wider["layers"][0]["mixer"]["left"]["mask"]["size"] = size + (1 if key == query - size else -1)
            assert row_errors(Z.forward(toks, w, wider)[-1:], want).max() > 0.1, "the planted key does not show"
            eng = engine_from(cfg, w, arm)
            for sizes in ([query + 1], [query, 1], [64]):
                eng.reserve_pool(160, 1)
                got = replay(eng, [[("a", c)] for c in portions(query + 1, sizes)], {"a": toks})["a"][-1:]
                assert row_errors(got, want).max() < (5e-5 if arm[1] == torch.float32 else 0.03), (key, query, sizes)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("channel", [False, True])
def test_far_memories_live_in_the_state(arm, channel):
    """A slowly forgetting layer: the first token's write is read 200 tokens later, however the tokens are cut.  The
    oracle without the first tokens is far off, so a state lost on the way would show."""
    d = delta(2, 1, 16, 16, 3)
    cfg = config(64, 100, [((None if channel else window(1, 1, 8, 8, 4, 4)), d, None)])
    w = Z.random_weights(cfg, seed=9)
    p = "l0.mix" if channel else "l0.mix.right"
    w[p + ".A_log"].fill_(-12.0)
    w[p + ".b"] *= 0.0
    w[p + ".b"][:, 0] = -1.0             # tokens with a positive first entry hardly write
    w["embed"][:, 0] = 6.0
    w["embed"][:3, 0] = -6.0             # ... and three tokens do
    toks = [0, 1, 2] + [3 + t % 97 for t in prompt(200, 100)]
    want = Z.forward(toks, w, cfg)[-1:]
    assert row_errors(Z.forward(toks[3:], w, cfg)[-1:], want).max() > 0.1, "the far memory does not show"
    eng = engine_from(cfg, w, arm)
    for sizes in ([203], [202, 1], [2, 64], [16, 1], [100, 3]):
        eng.reserve_pool(208, 1)
        got = replay(eng, [[("a", c)] for c in portions(203, sizes)], {"a": toks})["a"][-1:]
        assert row_errors(got, want).max() < (5e-5 if arm[1] == torch.float32 else 0.03), sizes


# ------------------------------------------------------------------ token trees
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide"])
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
            assert_rows(lg[r:r + 1].float().cpu(), Z.forward(p + [tk[i] for i in path], w, cfg)[-1:], arm[1])
            r += 1
    chosen = [paths[0][6], paths[1][3]]
    for s, p, t, path in zip(sids, pre, trees, chosen):
        eng.pool.commit_path(s, len(p), t.num_nodes, path)
    more = [prompt(3, cfg["vocab"], 7), prompt(1, cfg["vocab"], 8)]
    lg = eng.step([(s, m, list(range(len(m)))) for s, m in zip(sids, more)])
    want = [Z.forward(p + [tk[i] for i in path] + m, w, cfg)[-len(m):] for p, tk, path, m in zip(pre, toks, chosen, more)]
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
    want = [Z.greedy(p, w, cfg, new) for p in prompts]
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
    want = Z.greedy(p, w, cfg, new)
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
    assert want[0] == Z.greedy(prompts[0][0].tolist(), w, cfg, 20)
    for chunk in (None, 9):
        eng = engine_from(cfg, w, arm, num_pages=8, max_seq_len=64, max_seqs=4)
        assert [o["token_ids"] for o in eng.generate_batch(prompts, sp, prefill_chunk=chunk)] == want
        assert not eng.pool.resident()


@pytest.mark.parametrize("arm", ARMS)
def test_sampling_follows_the_distribution(arm):
    """How often first sampled tokens fall among the oracle's 20 likeliest at a high temperature."""
    from jetspec_b200 import SamplingParams
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    p = prompt(11, cfg["vocab"])
    eng = engine_from(cfg, w, arm, max_seqs=2)
    torch.manual_seed(0)
    n, temp = 60, 3.0
    draws = [eng.generate(torch.tensor([p]), SamplingParams(temp, 1))["token_ids"][0] for _ in range(n)]
    probs = torch.softmax(oracle_logits("mixed", cfg, w, p)[-1] / temp, -1)
    assert len(set(draws)) > 5
    top = set(probs.topk(20).indices.tolist())
    mass, hit = float(probs.topk(20).values.sum()), sum(t in top for t in draws) / n
    assert abs(hit - mass) < 4 * math.sqrt(mass * (1 - mass) / n) + 0.02


@pytest.mark.parametrize("arm", ARMS)
def test_draft_head_and_sampled_trees(arm):
    """A draft head conditioned on tapped layers (inside the round graph on the GPU) stays lossless; sampled rounds run."""
    from jetspec_b200 import DraftHeadTreeDrafter, RandomTreeDrafter, SamplingParams
    from jetspec_b200.models import DraftHeadModel, draft_head_config
    cfg = config(256, 211, [(window(4, 2, 32, 32, 19, 16), delta(4, 2, 24, 24, 4), moe(6, 2, 48, 40)),
                            (None, delta(3, 3, 16, 40, 4), moe(6, 3, 32)), (window(2, 2, 16, 16, 7, 8), delta(2, 2, 16, 16, 3), None)])
    w = margin_weights(cfg, 21)
    eng = engine_from(cfg, w, arm, max_seq_len=512, max_seqs=2)
    p = prompt(21, cfg["vocab"])
    want = Z.greedy(p, w, cfg, 8)
    head = DraftHeadModel.random_init(draft_head_config(eng.cfg, 1, 5, target_layer_ids=[0, 1, 2]), seed=1, dtype=arm[1], device=arm[0])
    kw = dict(tree_depth=4, tree_width=2, budget=8)
    d, t = DraftHeadTreeDrafter(head, eng.model, block_size=5), torch.tensor([p])
    assert eng.generate_tree(t, d, target_layer_ids=head.target_layer_ids, sampling_params=SamplingParams(0.0, 8), **kw)["token_ids"] == want
    out = eng.generate_tree(t, RandomTreeDrafter(cfg["vocab"], seed=2), sampling_params=SamplingParams(1.0, 8), **kw)["token_ids"]
    assert len(out) == 8 and all(0 <= x < cfg["vocab"] for x in out)


@pytest.mark.gpu
@pytest.mark.parametrize("case", ["mixed", "wide"])
def test_long_portions_run_their_branches_side_by_side(case):
    """From 512 rows on a portion's independent branches use two streams; short portions and single tokens do not."""
    from jetspec_b200.engine.hybrid_stack import FORK_MIN_TOKENS
    cfg, w, n = CASES[case], WEIGHTS[case], FORK_MIN_TOKENS + 90
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, ("cuda", torch.bfloat16))
    got = {}
    for name, sizes in (("whole", [n]), ("portions", [64, 1, 37]), ("both", [FORK_MIN_TOKENS, 1, 2])):
        eng.reserve_pool(n + 16, 1)
        got[name] = replay(eng, [[("a", c)] for c in portions(n, sizes)], {"a": toks})["a"]
    assert_rows(got["whole"], got["portions"].double(), torch.bfloat16)
    assert_rows(got["both"], got["portions"].double(), torch.bfloat16)
    assert_rows(got["whole"][-60:], oracle_logits(case, cfg, w, toks)[-60:], torch.bfloat16)


@pytest.mark.gpu
def test_experts_in_several_passes():
    """More (token, expert) pairs than one permutation takes: the tokens go through the experts in passes."""
    from jetspec_b200.engine.fast_round import FastRound
    cfg, w, arm = CASES["mixed"], WEIGHTS["mixed"], ("cuda", torch.bfloat16)
    toks = prompt(45, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(64, 1)
    FastRound.get(eng).stack.pass_rows = 14
    assert_rows(replay(eng, [[("a", 45)]], {"a": toks})["a"], oracle_logits("mixed", cfg, w, toks), arm[1])


# ------------------------------------------------------------------ checkpoints and the command line
def test_checkpoint_round_trip(tmp_path):
    from jetspec_b200.models import ZasipelForCausalLM, load_target
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    m = model_from(cfg, w, torch.bfloat16, "cpu")
    m.save_pretrained(str(tmp_path))
    assert json.load(open(tmp_path / "config.json")) == cfg
    from safetensors.torch import load_file, save_file
    t = load_file(str(tmp_path / "model.safetensors"))
    assert set(t) == set(w) and all(torch.equal(t[k].to(w[k].dtype), w[k]) for k in w)
    assert t["l0.mlp.table"].dtype == torch.int32
    m2, tok = load_target(str(tmp_path), device="cpu", dtype=torch.float32)
    assert tok is None and isinstance(m2, ZasipelForCausalLM) and m2.config == m.config
    assert all(torch.equal(a.float(), b.float()) for a, b in zip(m.state_dict().values(), m2.state_dict().values()))
    other = tmp_path / "other"           # never over a file that is mapped
    m.config.save_pretrained(str(other))
    for lost in ("l1.mlp.e2.up", "l0.mlp.table", "l1.mix.a2", "l0.mix.left.v.b"):
        save_file({k: v.clone() for k, v in t.items() if k != lost}, str(other / "model.safetensors"))
        with pytest.raises(KeyError):
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
