"""Karuzen against the plain statement in ``karuzen_oracle.py``: mechanisms, whole prompts, portions, mixed batches, reuse
of pages and slots, far keys, long decoding, and generation through the engine's own entry points."""
import json
import math
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))
import karuzen_oracle as K  # noqa: E402
from karuzen_cases import (ARMS, assert_rows, cases, config, dense, engine_from, mixer, model_from, moe, oracle_logits, portions,  # noqa: E402
                           prompt, replay, row_errors)

ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
CASES = cases()
WEIGHTS = {k: K.random_weights(c, seed=i) for i, (k, c) in enumerate(CASES.items())}


def rel(a, b):
    return ((a.double() - b.double()).abs().max() / b.double().abs().max().clamp(min=1e-9)).item()


# ------------------------------------------------------------------ mechanisms alone
def test_dynamic_tanh_block():
    from jetspec_b200.models.layers import DynamicTanh
    m = DynamicTanh(48)
    g = torch.Generator().manual_seed(0)
    w, b, a = torch.randn(48, generator=g), torch.randn(48, generator=g), 0.37
    with torch.no_grad():
        m.weight.copy_(w), m.bias.copy_(b), m.alpha.fill_(a)
    x = torch.randn(5, 48, generator=g) * 10
    assert rel(m(x), K.dynamic_tanh(x.double(), a, w.double(), b.double())) < 1e-6


def test_norm_puts_eps_inside_the_root():
    from jetspec_b200 import ops
    x, w = torch.full((1, 4), 1e-3), torch.ones(4)
    assert rel(ops.rmsnorm(x, w, 1e-6), K.rms_norm(x.double(), w.double(), 1e-6)) < 1e-6
    assert abs(float(ops.rmsnorm(x, w, 1e-6)[0, 0]) - 1 / math.sqrt(2)) < 1e-4


@pytest.mark.parametrize("vdim", [12, 20, 44])
def test_latent_attention_op_expands_keys_and_values(vdim):
    from jetspec_b200.ops import reference as ref
    m = mixer(3, 20, vdim, 28, 36, scale=0.31)
    g = torch.Generator().manual_seed(vdim)
    T, past = 6, 9
    uk, uv, c = torch.randn(60, 36, generator=g), torch.randn(3 * vdim, 36, generator=g), torch.randn(past + T, 36, generator=g)
    q = torch.randn(T, 3, 20, generator=g)
    pool, slots = torch.full((64, 64), 99.0), torch.randperm(64, generator=g)[:past + T].to(torch.int32)
    ref.latent_scatter(c, pool, slots)
    got = ref.latent_attention(q, uk, uv, pool, slots.view(1, -1), torch.tensor([0]), torch.tensor([0, T]), torch.tensor([past]), None,
                               m["scale"], True)
    k, v = (c @ uk.T).view(-1, 3, 20), (c @ uv.T).view(-1, 3, vdim)
    for i in range(T):
        for h in range(3):
            s = (k[:past + i + 1, h] @ q[i, h]) * m["scale"]
            p = torch.exp(s - s.max())
            assert rel(got[i].view(3, vdim)[h], (p / p.sum()) @ v[:past + i + 1, h]) < 1e-5


@pytest.mark.parametrize("top,scale,shared", [(1, 1.0, None), (3, 1.6, 24), (5, 0.5, None)])
def test_sigmoid_routed_experts_block(top, scale, shared):
    from jetspec_b200.models import RoutedExpertsConfig
    from jetspec_b200.models.layers import SigmoidMoE
    cfg = config(32, 16, [(mixer(1, 8, 8, 8, 8), moe(5, top, 20, scale, shared))])
    w = K.random_weights(cfg, seed=top, dtype=torch.float64)
    m = SigmoidMoE(RoutedExpertsConfig(5, top, scale, 20, shared or 0), 32)
    with torch.no_grad():
        m.router.weight.copy_(w["l0.mlp.router"]), m.correction.copy_(w["l0.mlp.correction"])
        for e in range(5):
            m.w_up[e].copy_(w[f"l0.mlp.e{e}.up"]), m.w_down[e].copy_(w[f"l0.mlp.e{e}.down"])
        if shared:
            m.shared_up.weight.copy_(w["l0.mlp.shared.up"]), m.shared_down.weight.copy_(w["l0.mlp.shared.down"])
            m.shared_gate.weight.copy_(w["l0.mlp.shared.sg"])
        h = torch.randn(9, 32, dtype=torch.float64)
        assert rel(m(h.float()), K.moe_mlp(h, w, "l0.mlp", cfg["layers"][0]["mlp"])) < 1e-5


def test_correction_chooses_but_does_not_weigh():
    """A large correction brings in an expert with a small score, which then gets the small weight."""
    from jetspec_b200.ops import reference as ref
    z = torch.tensor([[2.0, -3.0, 1.0, 0.0]])
    corr = torch.tensor([0.0, 5.0, 0.0, 0.0])
    w, idx = ref.sigmoid_route(z, corr, 2, 3.0)
    s = torch.sigmoid(z[0])
    assert idx[0].tolist() == [1, 0]
    assert torch.allclose(w[0], torch.stack((s[1], s[0])) / (s[0] + s[1]) * 3.0)


def test_gelu_mlp_block():
    from jetspec_b200.models.layers import GeluMLP
    m = GeluMLP(24, 40)
    w = {"p.gate": m.gate_proj.weight.detach().double(), "p.up": m.up_proj.weight.detach().double(),
         "p.down": m.down_proj.weight.detach().double()}
    h = torch.randn(7, 24) * 4
    with torch.no_grad():
        assert rel(m(h), K.dense_mlp(h.double(), w, "p")) < 1e-5


def test_layer_runs_of_a_loop():
    from jetspec_b200.models import KaruzenConfig
    for c in CASES.values():
        assert KaruzenConfig.from_dict(c).layer_runs() == K.schedule(c)
    c = KaruzenConfig.from_dict(CASES["mixed"])
    assert c.layer_runs() == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]
    assert c.latent_widths() == [36, 52, 36, 52, 36, 52]


def test_unknown_parts_are_refused():
    from jetspec_b200.models import KaruzenConfig, family_of
    bad = config(32, 16, [(mixer(1, 8, 8, 8, 8), None)])
    bad["layers"][0]["type"] = "something_else"
    with pytest.raises(ValueError):
        KaruzenConfig.from_dict(bad)
    with pytest.raises(ValueError):
        family_of({"architecture": "Unheard"})
    assert family_of({"architecture": "Karuzen"}).name == "karuzen"
    assert family_of({"architectures": ["Qwen3MoeForCausalLM"]}).name == "qwen3"


# ------------------------------------------------------------------ whole prompts, portions, decoding
@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", list(CASES))
def test_whole_prompt_and_residual_stream(arm, case):
    cfg, w = CASES[case], WEIGHTS[case]
    n = 150 if case == "wide" else 37
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(256, 2)
    got = replay(eng, [[("a", n)]], {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1])
    if arm[1] == torch.float32:         # the stream after every layer run
        streams = []
        K.forward(toks[:9], w, cfg, streams=streams)
        sid, runs = eng._new_seq_id(), list(range(len(streams)))
        eng.pool.reserve(sid, 9)
        _, hid, _ = eng._forward([sid], [torch.tensor(toks[:9])], [0], taps=runs)
        for r in runs[:-1]:
            assert rel(hid[:, r * cfg["width"]:(r + 1) * cfg["width"]].cpu(), streams[r]) < 2e-5, r


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case,sizes", [("mixed", [1]), ("mixed", [2]), ("mixed", [5, 2, 17]), ("routed", [3]), ("plain", [16, 1, 15]),
                                        ("ragged", [2, 31]), ("broad", [9, 1]), ("wide", [130, 1, 1, 2]), ("wide", [7])])
def test_portions_of_any_size_equal_the_whole(arm, case, sizes):
    """Prefill against token-by-token decoding and against portions cut inside and at the borders of pages."""
    cfg, w = CASES[case], WEIGHTS[case]
    n = 150 if case == "wide" else 37
    toks = prompt(n, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(192, 2)
    got = replay(eng, [[("a", c)] for c in portions(n, sizes)], {"a": toks})["a"]
    assert_rows(got, oracle_logits(case, cfg, w, toks), arm[1], sizes)


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide", "routed"])
def test_mixed_batches_equal_each_alone_and_reuse_pages(arm, case):
    """Unequal requests, portions beside single tokens, a request that sits steps out, and a pool so small that later
    requests take the pages and slot-map rows earlier ones gave back."""
    cfg, w = CASES[case], WEIGHTS[case]
    n = {"a": 37, "b": 5, "c": 150 if case == "wide" else 18, "d": 1, "e": 37}
    req = {k: prompt(v, cfg["vocab"], seed=i if k != "e" else 0) for i, (k, v) in enumerate(n.items())}
    long_c = [("c", 149)] if case == "wide" else [("c", 17)]
    sched = ([[("a", 16), ("b", 2)], [("b", 1), ("a", 1)] + long_c, [("a", 3), ("b", 1)], [("c", 1), ("a", 2), ("b", 1), ("d", 1)]]
             + [[("a", 1), ("e", 20)], [("e", 2), ("a", 13)]] + [[("a", 1), ("e", 1)]] + [[("e", 14)]])
    eng = engine_from(cfg, w, arm)
    tokens = 48 + 16 + (160 if case == "wide" else 32) + 16
    eng.reserve_pool(tokens, 4)
    got = replay(eng, sched, req)
    assert eng.pool.free_page_count == eng.pool.num_pages and not eng.pool.resident()
    for k in req:
        assert_rows(got[k], oracle_logits(case, cfg, w, req[k]), arm[1], k)
    assert_rows(got["e"], got["a"].double(), arm[1], "reused pages")


@pytest.mark.parametrize("arm", ARMS)
def test_long_decoding(arm):
    cfg, w = CASES["plain"], WEIGHTS["plain"]
    toks = prompt(140, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(144, 1)
    got = replay(eng, [[("a", 4)]] + [[("a", 1)]] * 136, {"a": toks})["a"]
    assert_rows(got, oracle_logits("plain", cfg, w, toks), arm[1])


# ------------------------------------------------------------------ far keys
def needle_model(key_pos, query_pos, n, width=64, vocab=130, wide=False):
    """One layer whose head 0 of the token at ``query_pos`` attends almost wholly to the one at ``key_pos``: two marker
    tokens share a direction that the query and key projections amplify.  Returns (cfg, weights, tokens)."""
    m = mixer(2, 72, 80, 16, 40, scale=1.0) if wide else mixer(2, 16, 16, 16, 40, scale=1.0)
    cfg = config(width, vocab, [(m, dense(32))])
    w = K.random_weights(cfg, seed=3)
    a, b = vocab - 1, vocab - 2                 # marker tokens: key and query
    w["embed"][:, :2] = 0.0
    w["embed"][a, 0] = 8.0
    w["embed"][b, 1] = 8.0
    for t in (".norm1.b", ".norm1.alpha"):
        w["l0" + t] = w["l0" + t] * (0.0 if t.endswith("b") else 1.0)
    w["l0.norm1"][:2] = 4.0
    # latent coordinate 0 carries the marker on both sides, head 0 multiplies them
    for name, col in (("l0.mix.dq", 1), ("l0.mix.dkv", 0)):
        w[name][0] = 0.0
        w[name][0, col] = 4.0
        w[name][1:, :2] = 0.0
    d = m["dim"]
    w["l0.mix.uq"][0], w["l0.mix.uk"][0] = 0.0, 0.0
    w["l0.mix.uq"][0, 0], w["l0.mix.uk"][0, 0] = 4.0, 4.0
    w["l0.mix.uq"][d:2 * d] *= 0.1
    toks = [t % (vocab - 2) for t in prompt(n, vocab)]
    toks[key_pos], toks[query_pos] = a, b
    return cfg, w, toks


FAR = [(0, 255), (0, 256), (1, 257), (15, 239), (16, 240), (17, 63), (31, 64), (32, 65), (63, 64), (64, 191), (127, 128), (254, 255)]


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("wide", [False, True])
def test_far_keys_at_page_and_tile_borders(arm, wide):
    """One key stands out of hundreds: the first tokens, both sides of a page's, a key tile's and a portion's edge, asked
    for from inside a prompt and by a decoded token.  The oracle without that key is far off, so a miss would show."""
    n = 260
    for key, query in FAR if not wide else FAR[::3]:
        cfg, w, toks = needle_model(key, query, n, wide=wide)
        toks = toks[:query + 1]
        want = K.forward(toks, w, cfg)[-1:]
        vis = torch.tril(torch.ones(query + 1, query + 1, dtype=torch.bool))
        vis[query, key] = False
        assert row_errors(K.forward(toks, w, cfg, visible=vis)[-1:], want).max() > 0.25, "the planted key does not show"
        eng = engine_from(cfg, w, arm)
        for sizes in ([query + 1], [query, 1], [64], [key, query + 1 - key] if key else [2, query - 1]):
            eng.reserve_pool(272, 1)
            got = replay(eng, [[("a", c)] for c in portions(query + 1, sizes)], {"a": toks})["a"][-1:]
            assert row_errors(got, want).max() < (5e-5 if arm[1] == torch.float32 else 0.05), (key, query, sizes)


# ------------------------------------------------------------------ generation
def margin_weights(cfg, seed):
    """Random weights whose greedy choice has a wide margin (bf16 rounding cannot flip it): small output projections, so
    that the stream stays near the token's embedding, plus a strong successor direction in the embedding."""
    w = K.random_weights(cfg, seed=seed)
    for k in w:
        if k.endswith(".o") or k.endswith(".down"):
            w[k] = (w[k] * 0.1).to(torch.bfloat16).double()
    return w


@pytest.mark.parametrize("arm", ARMS)
@pytest.mark.parametrize("case", ["mixed", "wide"])
def test_greedy_generation_through_every_entry_point(arm, case):
    from jetspec_b200 import LLM, RandomTreeDrafter, SamplingParams
    cfg = CASES[case]
    w = WEIGHTS[case] if arm[1] == torch.float32 else margin_weights(cfg, 11)
    prompts = [prompt(n, cfg["vocab"], seed=n) for n in (5, 23, 12)]
    new = 6
    want = [K.greedy(p, w, cfg, new) for p in prompts]
    t = [torch.tensor([p]) for p in prompts]
    sp = SamplingParams(0.0, new)
    eng = engine_from(cfg, w, arm, max_seq_len=512)
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


@pytest.mark.parametrize("arm", ARMS)
def test_batch_with_a_small_pool_evicts_and_restores(arm):
    from jetspec_b200 import SamplingParams
    cfg, w = CASES["mixed"], margin_weights(CASES["mixed"], 12)
    prompts = [torch.tensor([prompt(n, cfg["vocab"], seed=n)]) for n in (30, 28, 31)]
    sp = SamplingParams(0.0, 20)
    want = [engine_from(cfg, w, arm).generate(p, sp)["token_ids"] for p in prompts]
    for chunk in (None, 9):
        eng = engine_from(cfg, w, arm, num_pages=8, max_seq_len=64)
        assert [o["token_ids"] for o in eng.generate_batch(prompts, sp, prefill_chunk=chunk)] == want
        assert not eng.pool.resident()


@pytest.mark.parametrize("arm", ARMS)
def test_sampling_follows_the_distribution(arm):
    """How often first sampled tokens fall among the oracle's 20 likeliest at a high temperature."""
    from jetspec_b200 import SamplingParams
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    p = prompt(11, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    torch.manual_seed(0)
    n = 60
    draws = [eng.generate(torch.tensor([p]), SamplingParams(20.0, 1))["token_ids"][0] for _ in range(n)]
    probs = torch.softmax(oracle_logits("mixed", cfg, w, p)[-1] / 20.0, -1)
    assert len(set(draws)) > 5
    top = set(probs.topk(20).indices.tolist())
    mass, hit = float(probs.topk(20).values.sum()), sum(t in top for t in draws) / n
    assert abs(hit - mass) < 4 * math.sqrt(mass * (1 - mass) / n) + 0.02


@pytest.mark.parametrize("arm", ARMS)
def test_draft_head_and_sampled_trees(arm):
    """A draft head conditioned on tapped layer runs (inside the round graph on the GPU) stays lossless; sampled rounds run."""
    from jetspec_b200 import DraftHeadTreeDrafter, RandomTreeDrafter, SamplingParams
    from jetspec_b200.models import DraftHeadModel, draft_head_config
    mix = mixer(3, 40, 24, 56, 72)
    cfg = config(256, 211, [(mix, dense(160)), (mix, moe(6, 2, 48, 1.3, shared=40)), (mix, None)], loop=(0, 2, 2))
    w = margin_weights(cfg, 21)
    eng = engine_from(cfg, w, arm, max_seq_len=512)
    p = prompt(21, cfg["vocab"])
    want = K.greedy(p, w, cfg, 8)
    head = DraftHeadModel.random_init(draft_head_config(eng.cfg, 1, 5, target_layer_ids=[0, 1, 4]), seed=1, dtype=arm[1], device=arm[0])
    kw = dict(tree_depth=4, tree_width=2, budget=8)
    d = DraftHeadTreeDrafter(head, eng.model, block_size=5)
    t = torch.tensor([p])
    assert eng.generate_tree(t, d, target_layer_ids=head.target_layer_ids, sampling_params=SamplingParams(0.0, 8), **kw)["token_ids"] == want
    out = eng.generate_tree(t, RandomTreeDrafter(cfg["vocab"], seed=2), sampling_params=SamplingParams(1.0, 8), **kw)["token_ids"]
    assert len(out) == 8 and all(0 <= x < cfg["vocab"] for x in out)


@pytest.mark.gpu
def test_experts_in_several_passes(monkeypatch):
    """More (token, expert) pairs than one permutation launch takes: the tokens go through the experts in passes."""
    from jetspec_b200.engine import latent_stack
    monkeypatch.setattr(latent_stack, "MAX_SORT_PAIRS", 21)
    cfg, w, arm = CASES["mixed"], WEIGHTS["mixed"], ("cuda", torch.bfloat16)
    toks = prompt(37, cfg["vocab"])
    eng = engine_from(cfg, w, arm)
    eng.reserve_pool(64, 1)
    assert_rows(replay(eng, [[("a", 37)]], {"a": toks})["a"], oracle_logits("mixed", cfg, w, toks), arm[1])


def test_tree_visibility_matches_the_oracle():
    """A verify forward over a token tree: every node sees the prefix and its own ancestors only."""
    from jetspec_b200.tree import DraftTree
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    pre = prompt(19, cfg["vocab"])
    eng = engine_from(cfg, w, ("cpu", torch.float32))
    eng.reserve_pool(64, 1)
    sid = eng._new_seq_id()
    eng.step([(sid, pre, [])])
    parents, toks = [-1, 0, 0, 1, 2, 3], [7, 8, 9, 10, 11, 12]
    tree = DraftTree(torch.tensor(toks), torch.tensor(parents), torch.tensor([0, 1, 1, 2, 2, 3]), 6)
    eng.pool.reserve(sid, 19 + 6)
    lg, _, _ = eng._forward([sid], [tree.token_ids], [19], trees=[tree])
    for i in range(6):
        path, j = [], i
        while j >= 0:
            path.append(toks[j])
            j = parents[j]
        assert_rows(lg[i:i + 1], K.forward(pre + path[::-1], w, cfg)[-1:], torch.float32)


# ------------------------------------------------------------------ checkpoints and the command line
def test_checkpoint_round_trip(tmp_path):
    from jetspec_b200.models import KaruzenForCausalLM, load_target
    cfg, w = CASES["mixed"], WEIGHTS["mixed"]
    m = model_from(cfg, w, torch.bfloat16, "cpu")
    m.save_pretrained(str(tmp_path))
    saved = json.load(open(tmp_path / "config.json"))
    assert saved == cfg
    from safetensors.torch import load_file
    t = load_file(str(tmp_path / "model.safetensors"))
    assert set(t) == set(w) and all(torch.equal(t[k].double().view(w[k].shape), w[k]) for k in w)
    m2, tok = load_target(str(tmp_path), device="cpu", dtype=torch.float32)
    assert tok is None and isinstance(m2, KaruzenForCausalLM)
    assert all(torch.equal(a.float(), b) for a, b in zip(m.parameters(), m2.parameters()))
    assert m2.lm_head.weight.data_ptr() == m2.model.embed_tokens.weight.data_ptr()
    del t["l1.mlp.e2.up"]
    from safetensors.torch import save_file
    save_file(t, str(tmp_path / "model.safetensors"))
    with pytest.raises(KeyError):
        load_target(str(tmp_path), device="cpu", dtype=torch.float32)


@pytest.mark.parametrize("arm", ARMS)
def test_trace_replay_command(arm, tmp_path):
    """The command: steps on standard input, logits in files, ``done`` lines, pages given back at ``end``."""
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
            got = torch.from_numpy(np.fromfile(path, dtype="<f4").reshape(-1, cfg["vocab"]))
            assert_rows(got, rows, arm[1], i)
