"""Kernels of the latent-attention stack against plain fp32 PyTorch statements of the same op."""
import math

import pytest
import torch

pytestmark = pytest.mark.gpu
DEV = "cuda"


@pytest.fixture(scope="module")
def ext():
    from jetspec_b200.ops import cuda_ext
    cuda_ext.load()
    return cuda_ext


def bf(*shape, scale=1.0, seed=0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(torch.bfloat16).to(DEV)


def close(a, b, tol=8e-3):
    err = (a.float() - b.float()).abs().max().item() / max(b.float().abs().max().item(), 1e-6)
    assert err < tol, err


def gelu(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


@pytest.mark.parametrize("M,K,n_raw,ff,bn,split,deep", [
    (1, 192, 128, 64, 128, 1, 0), (130, 256, 256, 192, 128, 1, 1), (17, 512, 128, 320, 128, 4, 2), (33, 328, 128, 128, 128, 2, 1),
    (65, 512, 256, 64, 128, 3, 1), (300, 256, 128, 192, 256, 1, 0), (64, 256, 256, 0, 128, 2, 1)])
@pytest.mark.parametrize("gelu_act", [True, False])
def test_fused_input_projection(ext, M, K, n_raw, ff, bn, split, deep, gelu_act):
    """fp32 columns, then activated columns; with 256-column tiles the boundary may fall inside a tile."""
    cols = ff if gelu_act else (ff + 127) // 128 * 128
    x, wr = bf(M, K), bf(n_raw, K, scale=K ** -0.5, seed=1)
    wa, wb = bf(cols, K, scale=K ** -0.5, seed=2), bf(cols, K, scale=K ** -0.5, seed=3)
    if gelu_act:
        w = torch.cat((wr, torch.cat((wa.view(-1, 64, K), wb.view(-1, 64, K)), 1).reshape(-1, K)))
    else:
        w = torch.cat((wr, wa))
    raw = torch.full((M, n_raw), 7.0, device=DEV)
    act = torch.full((M, cols + 8), 7.0, dtype=torch.bfloat16, device=DEV)
    ext.gemm_inproj(x, w.contiguous(), raw, n_raw, act[:, :cols] if cols else None, gelu_act, bn=bn, split=split, deep=deep)
    ext.check_status(DEV)
    close(raw, x.float() @ wr.float().t(), 1e-5)
    if cols:
        a, b = x.float() @ wa.float().t(), x.float() @ wb.float().t()
        close(act[:, :cols], gelu(a) * b if gelu_act else torch.relu(a) ** 2)
        assert (act[:, cols:] == 7).all()


@pytest.mark.parametrize("M,N,K,bn,split,deep", [
    (1, 192, 264, 128, 1, 0), (129, 328, 512, 128, 1, 1), (20, 256, 1024, 128, 4, 1), (20, 256, 1024, 128, 3, 2),
    (300, 512, 256, 256, 1, 1), (300, 512, 256, 256, 1, 3)])
@pytest.mark.parametrize("with_norm,with_emb", [(False, False), (True, False), (True, True)])
def test_output_projection_on_the_fp32_stream(ext, M, N, K, bn, split, deep, with_norm, with_emb):
    a, w, e = bf(M, K), bf(N, K, scale=K ** -0.5, seed=1), bf(M, N, seed=2)
    g = torch.Generator().manual_seed(5)
    x = (torch.randn(M, N, generator=g) * 30).to(DEV)
    nw, nb = torch.randn(N, generator=g).to(DEV), torch.randn(N, generator=g).to(DEV)
    want = x + a.float() @ w.float().t() + (e.float() if with_emb else 0)
    h = torch.zeros(M, N, dtype=torch.bfloat16, device=DEV)
    ext.gemm_resid32(a, w, x, norm=(nw, nb, 0.37) if with_norm else None, h=h if with_norm else None, emb=e if with_emb else None,
                     bn=bn, split=split, deep=deep)
    ext.check_status(DEV)
    close(x, want, 1e-6)
    if with_norm:
        close(h, torch.tanh(0.37 * want) * nw + nb)


@pytest.mark.parametrize("M,H,K,N,shared", [(3, 5, 40, 128, False), (200, 3, 24, 72, False), (130, 4, 128, 512, False),
                                            (70, 6, 192, 40, True), (1, 2, 64, 8, False)])
def test_batched_products_over_heads(ext, M, H, K, N, shared):
    """K per head below, at and off the 64-column boxes: a box that reaches into the next head must not count it."""
    a = bf(M, K if shared else H * K)
    w = bf(H * N, K, scale=K ** -0.5, seed=1)
    out = torch.full((M, H * N + 8), 3.0, dtype=torch.bfloat16, device=DEV)
    ext.gemm_batched(a, w, out, H, N, K, 0 if shared else K, N, out.stride(0))
    ext.check_status(DEV)
    for h in range(H):
        ah = a.float() if shared else a[:, h * K:(h + 1) * K].float()
        close(out[:, h * N:(h + 1) * N], ah @ w[h * N:(h + 1) * N].float().t())
    assert (out[:, H * N:] == 3).all()


def latent_case(H, R, counts, pasts, tree, seed=0, dtype=torch.bfloat16, page=16):
    """Query rows, a pool with scattered pages (every slot that is not a key of the batch holds a huge row) and the
    expected attention per row, in double precision."""
    from jetspec_b200.runtime.kv_pool import latent_row_width
    g = torch.Generator().manual_seed(seed)
    Rp, B, T = latent_row_width(R), len(counts), sum(counts)
    lens = [c + p for c, p in zip(counts, pasts)]
    max_len = (max(lens) + page - 1) // page * page
    pages = [(n + page - 1) // page for n in lens]
    perm = torch.randperm(sum(pages) + 5, generator=g)
    S = (sum(pages) + 5) * page
    pool = torch.full((S, Rp), 1e4, dtype=dtype)
    slot_map = torch.zeros(B + 2, max_len, dtype=torch.int32)
    rows = torch.randperm(B + 2, generator=g)[:B].to(torch.int32)
    q = torch.zeros(T, H, Rp, dtype=dtype)
    q[:, :, :R] = torch.randn(T, H, R, generator=g).to(dtype)
    used, at = 0, 0
    scale = R ** -0.5
    want = torch.zeros(T, H, Rp, dtype=torch.float64)
    W = max(1, (max(counts) + 31) // 32)
    bits = torch.zeros(T, W, dtype=torch.int64)
    for b in range(B):
        ids = torch.cat([perm[used + k] * page + torch.arange(page) for k in range(pages[b])])
        if tree:       # a committed tree path leaves the window's slots permuted
            w = ids[pasts[b]:lens[b]]
            ids[pasts[b]:lens[b]] = w[torch.randperm(len(w), generator=g)]
        used += pages[b]
        slot_map[rows[b], : len(ids)] = ids.to(torch.int32)
        c = torch.zeros(lens[b], Rp, dtype=dtype)
        c[:, :R] = torch.randn(lens[b], R, generator=g).to(dtype)
        pool[ids[: lens[b]]] = c
        for i in range(counts[b]):
            # make one key stand out: sometimes the first, sometimes the own, sometimes in between
            tgt = [0, pasts[b] + i, int(torch.randint(0, pasts[b] + 1, (1,), generator=g))][i % 3]
            q[at + i, :, :R] += (2.0 * c[tgt, :R].float()).to(dtype)
        qs = q[at:at + counts[b]].double()
        sc = torch.einsum("nhr,lr->nhl", qs, c.double()) * scale
        vis = torch.ones(counts[b], lens[b], dtype=torch.bool)
        if tree:
            anc = torch.rand(counts[b], counts[b], generator=g) < 0.3
            anc |= torch.eye(counts[b], dtype=torch.bool)
            vis[:, pasts[b]:] = anc
            for i in range(counts[b]):
                for j in range(counts[b]):
                    if anc[i, j]:
                        bits[at + i, j >> 5] |= 1 << (j & 31)
        else:
            vis[:, pasts[b]:] = torch.tril(torch.ones(counts[b], counts[b], dtype=torch.bool))
        p = torch.softmax(sc.masked_fill(~vis[:, None], float("-inf")), -1)
        want[at:at + counts[b]] = torch.einsum("nhl,lr->nhr", p, c.double())
        at += counts[b]
    bits = torch.where(bits >= 2 ** 31, bits - 2 ** 32, bits).to(torch.int32)
    cu = torch.tensor([0] + list(torch.tensor(counts).cumsum(0)), dtype=torch.int32)
    d = lambda t: t.to(DEV)
    return dict(q=d(q).view(T * H, Rp), pool=d(pool), slot_map=d(slot_map), rows=d(rows), cu=d(cu),
                past=d(torch.tensor(pasts, dtype=torch.int32)), bits=d(bits) if tree else None, scale=scale,
                want=d(want).view(T * H, Rp), max_q=max(counts), max_keys=max(lens))


CASES = [(6, 104, [1], [300]), (3, 72, [1, 1, 1, 1], [0, 63, 64, 200]), (5, 40, [130, 2, 33], [0, 65, 31]), (16, 320, [3, 1], [127, 500]),
         (32, 512, [1, 1], [600, 15]), (12, 512, [40, 7], [100, 0]), (128, 256, [2, 1], [70, 129]), (1, 64, [200], [57]),
         (7, 192, [19], [1000])]


@pytest.mark.parametrize("H,R,counts,pasts", CASES)
@pytest.mark.parametrize("splits", [1, 3])
@pytest.mark.parametrize("tree", [False, True])
def test_latent_attention_tensor_cores(ext, H, R, counts, pasts, splits, tree):
    c = latent_case(H, R, counts, pasts, tree)
    out = ext.latent_attention_rows(c["q"], c["pool"], H, c["slot_map"], c["rows"], c["cu"], c["past"], c["bits"], c["scale"],
                                    not tree, c["max_q"], splits=splits, impl="tc")
    ext.check_status(DEV)
    close(out, c["want"])


@pytest.mark.parametrize("H,R,counts,pasts", CASES + [(2, 700, [5, 1], [40, 9])])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 8e-3)])
@pytest.mark.parametrize("tree", [False, True])
def test_latent_attention_plain_cores(ext, H, R, counts, pasts, dtype, tol, tree):
    c = latent_case(H, R, counts, pasts, tree, dtype=dtype)
    out = ext.latent_attention_rows(c["q"], c["pool"], H, c["slot_map"], c["rows"], c["cu"], c["past"], c["bits"], c["scale"],
                                    not tree, c["max_q"], impl="simt")
    ext.check_status(DEV)
    close(out, c["want"], tol)


@pytest.mark.parametrize("T,E,k", [(5, 18, 3), (300, 6, 2), (9, 200, 8), (40, 700, 1), (3, 4, 4)])
def test_sigmoid_routing_and_shared_gate(ext, T, E, k):
    from jetspec_b200.ops import reference as ref
    g = torch.Generator().manual_seed(T)
    z = (torch.randn(T, E + 3, generator=g) * 2).to(DEV)
    corr = torch.randn(E, generator=g).to(DEV)
    act = bf(T, 40)
    before = act.clone()
    wts, idx = ext.sigmoid_route(z, corr, k, 1.7, gate_col=E + 1, act=act[:, :32])
    wr, ir = ref.sigmoid_route(z[:, :E], corr, k, 1.7)
    assert torch.equal(idx.long(), ir)
    close(wts, wr, 1e-5)
    close(act[:, :32], before[:, :32].float() * torch.sigmoid(z[:, E + 1:E + 2]))
    assert torch.equal(act[:, 32:], before[:, 32:])


@pytest.mark.parametrize("qr,kr", [(56, 72), (2200, 40), (300, 2100)])
def test_latent_norms_go_to_the_query_and_to_the_pool(ext, qr, kr):
    T, eps, qp, Rp = 9, 1e-3, (qr + 15) // 8 * 8, (kr + 127) // 64 * 64
    ld = qr + kr + 5
    g = torch.Generator().manual_seed(1)
    proj = (torch.randn(T, ld, generator=g) * 0.05).to(DEV)
    qw, kw = bf(qr, seed=2), bf(kr, seed=3)
    cq = torch.full((T, qp), 5.0, dtype=torch.bfloat16, device=DEV)
    pool = torch.full((40, Rp), 5.0, dtype=torch.bfloat16, device=DEV)
    slots = torch.randperm(40, generator=g)[:T].to(torch.int32).to(DEV)
    lib, p = ext.load(), ext._p
    ext._check(lib.js_latent_post(p(proj), ld, qr, kr, p(qw), p(kw), ext.ctypes.c_float(eps), p(cq), qp, p(pool), Rp, 40, p(slots), T,
                                  p(ext.status_word(DEV)), 0, ext._stream()), "js_latent_post")
    ext.check_status(DEV)
    rms = lambda x, w: x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * w.float()
    close(cq[:, :qr], rms(proj[:, :qr], qw))
    close(pool[slots.long(), :kr], rms(proj[:, qr:qr + kr], kw))
    assert (cq[:, qr:] == 0).all() and (pool[slots.long(), kr:] == 0).all()
    rest = torch.ones(40, dtype=torch.bool, device=DEV)
    rest[slots.long()] = False
    assert (pool[rest] == 5).all()


@pytest.mark.parametrize("T,W,k", [(3, 192, 2), (200, 4096, 8)])
def test_expert_combine_with_embedding_and_norm(ext, T, W, k):
    g = torch.Generator().manual_seed(2)
    ys, emb = bf(T * k, W), bf(T, W, seed=1)
    inv = torch.randperm(T * k, generator=g).to(torch.int32).to(DEV)
    rw = torch.rand(T * k, generator=g).to(DEV)
    x, nw, nb = torch.randn(T, W, generator=g).to(DEV), torch.randn(W, generator=g).to(DEV), torch.randn(W, generator=g).to(DEV)
    h = torch.zeros(T, W, dtype=torch.bfloat16, device=DEV)
    r = inv.long().view(T, k)
    want = x + (ys.float()[r] * rw[r][..., None]).sum(1) + emb.float()
    lib, p = ext.load(), ext._p
    ext._check(lib.js_combine_dyt(p(ys), W, p(inv), p(rw), k, p(emb), p(x), p(h), W, p(nw), p(nb), ext.ctypes.c_float(0.6), T, W, 0,
                                  ext._stream()), "js_combine_dyt")
    close(x, want, 1e-5)
    close(h, torch.tanh(0.6 * want) * nw + nb)


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-6), (torch.bfloat16, 8e-3)])
def test_unfused_elementwise_ops(dtype, tol):
    from jetspec_b200 import ops
    from jetspec_b200.ops import reference as ref
    g = torch.Generator().manual_seed(4)
    x = (torch.randn(7, 100, generator=g) * 3).to(DEV)
    a, w, b = (torch.randn(s, generator=g).to(dtype).to(DEV) for s in ((), (100,), (100,)))
    for od in (torch.float32, torch.bfloat16):
        close(ops.dynamic_tanh(x, a, w, b, od), ref.dynamic_tanh(x, a, w, b, torch.float32), 1e-6 if od == torch.float32 else 8e-3)
    xx, yy = x.to(dtype), x.flip(0).to(dtype)
    close(ops.gelu_tanh_mul(xx, yy), ref.gelu_tanh_mul(xx.float(), yy.float()), tol)
    close(ops.relu_squared(xx), ref.relu_squared(xx.float()), tol)
