"""Kabulix kernels and the model on the GPU against plain fp64 PyTorch (kabulix_oracle.py and the formulas below)."""
import math

import pytest
import torch
import torch.nn.functional as F

import kabulix_oracle as O

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
BF = torch.bfloat16


@pytest.fixture(autouse=True)
def _true_fp32():
    """Library products in fp32 proper, whatever a test before this one has chosen."""
    before = torch.get_float32_matmul_precision()
    torch.set_float32_matmul_precision("highest")
    yield
    torch.set_float32_matmul_precision(before)


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-30)).item()


def tol(dtype, scale=1.0):
    return scale * (4e-6 if dtype == torch.float32 else 6e-3)


def rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).cuda()


def tokens(n, seed, vocab=300):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ---------------------------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,k", [(5, 64, 2), (3, 66, 1), (7, 2048, 6), (2, 6144, 3), (4, 1030, 4), (300, 256, 2)])
def test_prenorm_sum_and_norm(dtype, T, W, k):
    """Sum of a gated addend and a token's weighted experts, fp32 stream, norm; all rows and wanted rows only."""
    from trainscale_b200.ops import stream
    x, w = rnd(T, W, seed=1), rnd(W, seed=3, scale=0.3)
    y = rnd(T, W + (8 if W % 4 == 0 else 3), seed=2, dtype=dtype, scale=3.0)[:, :W]
    logits, wts = rnd(T, 5, seed=4), torch.rand(T, k, generator=torch.Generator().manual_seed(5)).cuda()
    e = rnd(T * k + 9, W, seed=6, dtype=dtype)
    dest = torch.randperm(T * k + 9, generator=torch.Generator().manual_seed(7))[:T * k].int().cuda()
    sel = i32(*[T - 1, 0][:T])
    for gate in (None, logits[:, 3]):
        for experts in (None, (e, dest, wts), (e, None, wts)):
            want = x.double() + y.double() * (1.0 if gate is None else torch.sigmoid(gate.double())[:, None])
            if experts is not None:
                rows = torch.arange(T * k, device="cuda") if experts[1] is None else dest.long()
                want = want + (e[rows].double().view(T, k, W) * wts.double()[..., None]).sum(1)
            got, h = stream.prenorm(x, y, gate, experts, w, 1e-4, dtype)
            assert rel(got, want) < 2e-6 and rel(h, O.norm1p(want, w.double(), 1e-4)) < tol(dtype) and h.dtype == dtype
            assert rel(stream.prenorm_final(x, y, gate, experts, w, 1e-4, sel, dtype), O.norm1p(want, w.double(), 1e-4)[sel.long()]) < tol(dtype)
    assert stream.prenorm_final(x, y, None, None, w, 1e-4, sel[:0], dtype).shape == (0, W)
    tok, table = torch.tensor([3, 49, 0, 3, 7], device="cuda"), rnd(50, W, seed=8, dtype=dtype)
    got, h = stream.prenorm_embed(tok, table, w, 1e-4)
    assert torch.equal(got, table[tok].float()) and rel(h, O.norm1p(table[tok].double(), w.double(), 1e-4)) < tol(dtype)


# ---------------------------------------------------------------------------------------------- gated products, experts
def packed(gate, up):
    from trainscale_b200.ops import grouped
    w = torch.zeros(2 * grouped.glu_width(gate.shape[0]), gate.shape[1], dtype=gate.dtype, device="cuda")
    for i, t in enumerate((gate, up)):
        grouped.GluRows(w, gate.shape[0], i).copy_(t)
    return w


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,ff,K", [(1, 40, 64), (9, 16, 200), (20, 17, 128), (31, 500, 2048), (70, 300, 64), (257, 33, 72), (600, 512, 256),
                                    (2500, 1030, 192), (5, 9, 21), (40, 30, 50)])
def test_gated_products(dtype, M, ff, K):
    from trainscale_b200.ops import gemm, grouped
    x = rnd(M, K, seed=1, dtype=dtype)
    g, u = rnd(ff, K, seed=2, dtype=dtype, scale=2 * K ** -0.5), rnd(ff, K, seed=3, dtype=dtype, scale=K ** -0.5)
    w = packed(g, u)
    zg, zu = x.double() @ g.double().t(), x.double() @ u.double().t()
    for act, want in ((grouped.ACT_SILU_GLU, F.silu(zg) * zu), (grouped.ACT_GELU_GLU, O.gelu_tanh(zg) * zu)):
        y = gemm.serve_linear(x, w, act=act)
        assert y.shape == (M, grouped.glu_width(ff)) and rel(y[:, :ff], want) < tol(dtype, 1.5) and (y[:, ff:] == 0).all()


def test_gated_product_of_large_values():
    """The sigmoid saturates without overflow on either side."""
    from trainscale_b200.ops import gemm, grouped
    for M, dtype in ((4, BF), (300, BF), (4, torch.float32)):
        x = torch.full((M, 64), 40.0, dtype=dtype, device="cuda")
        g = torch.cat([torch.full((16, 64), 5.0), torch.full((16, 64), -5.0)]).to(dtype).cuda()
        u = torch.full((32, 64), 0.5, dtype=dtype, device="cuda")
        for act in (grouped.ACT_SILU_GLU, grouped.ACT_GELU_GLU):
            y = gemm.serve_linear(x, packed(g, u), act=act).float()
            assert torch.isfinite(y).all() and rel(y[:, :16], torch.full((M, 16), 12800.0 * 1280.0)) < 0.01 and (y[:, 16:].abs() < 1e-3).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,top,count,keep,ff", [
    (1, 64, 12, 3, 4, 2, 24), (9, 96, 12, 3, 4, 2, 40), (32, 64, 16, 8, 4, 2, 17), (33, 64, 8, 4, 8, 5, 136), (64, 64, 40, 4, 5, 1, 64),
    (300, 96, 12, 3, 4, 3, 40), (500, 128, 6, 2, 1, 1, 200), (90, 50, 6, 2, 6, 3, 17), (9, 50, 6, 2, 3, 3, 17), (200, 64, 256, 8, 8, 4, 32),
    (20, 64, 1024, 32, 64, 9, 8), (70, 64, 99, 5, 33, 2, 16)])
def test_grouped_router_and_gated_experts(dtype, T, W, E, top, count, keep, ff):
    """Router, plan and both expert products against a loop over slots; decode-sized and prompt-sized batches."""
    from trainscale_b200.ops import gemm, grouped, moe
    x, router = rnd(T, W, seed=1, dtype=dtype), rnd(-(-(E + 1) // 8) * 8, W, seed=2, dtype=dtype, scale=2 / math.sqrt(W))
    g, u, d = (rnd(E, *s, seed=3 + i, dtype=dtype, scale=s[1] ** -0.5) for i, s in enumerate(((ff, W), (ff, W), (W, ff))))
    w_in = torch.stack([packed(g[e], u[e]) for e in range(E)])
    w_down = torch.zeros(E, W, grouped.glu_width(ff), dtype=dtype, device="cuda")
    w_down[:, :, :ff] = d
    logits = gemm.serve_linear(x, router, torch.float32)
    y, dest, w = moe.routed_experts(x, logits, w_in, w_down, moe.Router(E, top, True, count, keep), grouped.ACT_SILU_GLU)
    idx, ws = O.group_routing(logits[:, :E].double().cpu(), top, count, keep)
    assert rel(w, ws) < 3e-6
    y = y[dest.long()] if dest is not None else y
    rows, slots = x.repeat_interleave(top, 0).double(), idx.reshape(-1).cuda()
    want = torch.empty(T * top, W, dtype=torch.float64, device="cuda")
    for e in slots.unique().tolist():
        at = (slots == e).nonzero().flatten()
        a = F.silu(rows[at] @ g[e].double().t()) * (rows[at] @ u[e].double().t())
        want[at] = a @ d[e].double().t()
    assert rel(y, want) < tol(dtype, 2.0)


def test_router_without_group_limit_and_ties():
    """Equal scores go to the lower expert; softmax routing is unchanged by the row stride."""
    from trainscale_b200.ops import moe
    for fn in (lambda z, r: moe._topk_raw(z, r)[1], lambda z, r: moe._route_decode(z, r)[1]):
        z = torch.zeros(3, 24, device="cuda")
        got = fn(z, moe.Router(16, 2, True, 4, 1))
        if got.dim() == 1:                                       # expert-sorted slots: expert 0 of every token, then expert 1
            assert got.tolist() == [0, 2, 4, 1, 3, 5]
        else:
            assert got.tolist() == [[0, 1]] * 3
    z = rnd(50, 20, seed=1)
    a = moe._topk_raw(z[:, :12], moe.Router(12, 3, True))
    b = moe._topk_raw(z[:, :12].contiguous(), moe.Router(12, 3, True))
    assert torch.equal(a[0], b[0]) and torch.equal(a[1], b[1])
    s, idx = torch.softmax(z[:, :12].double(), -1).topk(3, -1)
    assert torch.equal(a[1].long(), idx) and rel(a[0], s / s.sum(-1, keepdim=True)) < 3e-6


# ---------------------------------------------------------------------------------------------- grouped-query attention
def visible(mask, n, device="cpu"):
    return (O.chunk_mask(n, mask.size) if mask.chunked else O.window_mask(n, mask.size, mask.keep)).to(device)


SHAPES = [  # H, G, dim, vdim, rot
    (5, 1, 96, 96, 40), (8, 2, 128, 128, 64), (4, 4, 64, 64, 64), (5, 5, 40, 72, 12), (24, 1, 80, 48, 16), (3, 1, 20, 12, 6),
    (4, 2, 18, 30, 18), (2, 1, 256, 128, 32), (2, 2, 200, 256, 0)]


def shape_of(H, G, D, V, rot, mask, **kw):
    from trainscale_b200.ops.window_attention import WindowShape
    return WindowShape(H, G, D, V, rot, mask.size, D ** -0.5 * 1.3, mask.keep, mask.chunked, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,rot", SHAPES)
@pytest.mark.parametrize("biased,normed,turned,shared", [(True, True, True, True), (False, True, True, False), (True, False, False, True),
                                                         (False, False, True, False), (False, False, False, False), (False, True, False, True)])
def test_prepare_bias_norms_pairs_and_cache_write(dtype, H, G, D, V, rot, biased, normed, turned, shared):
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import KeyMask
    V, rot = (D if shared else V), (rot if turned else 0)
    s = shape_of(H, G, D, V, rot, KeyMask(9), pairs=True, values_are_keys=shared)
    T, pad = 37, 8 + (-(s.q_width + s.kv_width)) % 8
    proj = rnd(T, s.q_width + s.kv_width + pad, seed=1, dtype=dtype)
    before = proj.clone()
    bias = rnd(s.q_width + G * D, seed=6) if biased else None
    qn, kn = (rnd(D, seed=2), rnd(D, seed=3)) if normed else (None, None)
    pos = torch.randint(0, 5000, (T,), generator=torch.Generator().manual_seed(4)).int().cuda()
    slots = torch.randperm(64, generator=torch.Generator().manual_seed(5))[:T].cuda()
    r = {"dims": rot, "base": 1000.0, "scaling": O.SCALING}
    cache = torch.full((8, 8, s.row_width), 3.0, dtype=dtype, device="cuda")
    cs = wa.angles(O.frequencies(r).float().cuda(), pos, O.magnitude(r)) if rot else None
    wa.prepare(proj, s, qn, kn, 1e-5, cs, slots, cache, bias)
    qw, kw = s.q_width, G * D
    x = before.double().cpu()
    if biased:
        x[:, :qw + kw] += bias.double().cpu()

    def changed(y, w):
        y = O.rms(y, 1e-5) * w.double().cpu() if w is not None else y
        return (O.rotate_pairs(y, pos.cpu(), r) if rot else y).reshape(T, -1)

    loose = 5e-5 if dtype == torch.float32 else 6e-3            # fp32 angles of positions up to 5000
    assert rel(proj[:, :qw], changed(x[:, :qw].reshape(T, H, D), qn)) < loose
    assert rel(proj[:, qw:qw + kw], changed(x[:, qw:qw + kw].reshape(T, G, D), kn)) < loose
    if shared:
        assert rel(proj[:, qw + kw:qw + s.kv_width], x[:, qw:qw + kw]) < tol(dtype)
    else:
        assert torch.equal(proj[:, qw + kw:qw + s.kv_width], before[:, qw + kw:qw + s.kv_width])
    assert torch.equal(proj[:, qw + s.kv_width:], before[:, qw + s.kv_width:])
    rows = cache.view(-1, s.row_width)[slots]
    assert torch.equal(rows[:, :s.kv_width], proj[:, qw:qw + s.kv_width]) and rows[:, s.kv_width:].abs().sum() == 0
    other = torch.ones(64, dtype=torch.bool)
    other[slots.cpu()] = False
    assert (cache.view(-1, s.row_width)[other.cuda()] == 3).all()


MASKS = [(50, 4, False), (1, 1, False), (5, 40, False), (130, 16, False), (300, 700, False), (129, 0, False), (40, 0, True), (128, 0, True),
         (1, 0, True), (700, 0, True)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,rot", SHAPES)
@pytest.mark.parametrize("size,keep,chunked", MASKS)
@pytest.mark.parametrize("gated", [0, 1, 2])
def test_attend_rows_masks_and_gates(dtype, H, G, D, V, rot, size, keep, chunked, gated):
    """Single query rows against scattered pages.  The keys on both sides of every edge of what a row sees are made to stand
    out, one edge at a time."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import KeyMask
    mask, bs = KeyMask(size, keep, chunked), 16
    s = shape_of(H, G, D, V, rot, mask)
    lens = [1, 2, size, size + 1, size + keep + 1, 2 * size + 3, 700, 701, 1500]
    n, nb = len(lens), 1500 // bs + 100
    perm = torch.randperm(n * nb + 3, generator=torch.Generator().manual_seed(1))[:n * nb].view(n, nb).int()
    cache = rnd(n * nb + 3, bs, s.row_width, seed=2, dtype=dtype)
    q = rnd(n, s.q_width + 16 + (-s.q_width) % 8, seed=3, dtype=dtype)
    flat = cache.view(-1, s.row_width)
    slot = lambda b, j: int(perm[b, j // bs]) * bs + j % bs      # noqa: E731
    for b, L in enumerate(lens):
        lo = mask.first(L - 1)
        for j, f in ((lo, 1.5), (lo - 1, 3.0), (min(keep, lo) - 1, 1.5), (keep, 3.0 if keep < lo else 0.0)):
            if 0 <= j < L and f:
                flat[slot(b, j), :D] = q[b, :D] * f
    gate = {0: None, 1: rnd(n, H + 3, seed=7, dtype=dtype)[:, :H], 2: rnd(n, s.out_width + 8, seed=8, dtype=dtype)[:, :s.out_width]}[gated]
    out = torch.zeros(n, s.out_width + 8, dtype=dtype, device="cuda")
    wa.attend_rows(q, s, cache, perm.cuda(), torch.arange(n, dtype=torch.int32, device="cuda"), i32(*lens), max(lens), out[:, :s.out_width], 0.75, gate)
    for b, L in enumerate(lens):
        rows = flat[torch.tensor([slot(b, j) for j in mask.positions(L - 1)]).cuda()].double()
        k, v = rows[:, :G * D].view(-1, G, D), rows[:, G * D:s.kv_width].view(-1, G, V)
        want = O.attend(q[b:b + 1, :s.q_width].double().view(1, H, D), k, v, s.scale, torch.ones(1, len(rows), dtype=torch.bool, device="cuda")) * 0.75
        if gated:
            want = want * torch.sigmoid(gate[b].double()).view(1, H, -1)
        assert rel(out[b, :s.out_width], want.reshape(-1)) < tol(dtype, 1.5), (b, L)
    assert out[:, s.out_width:].abs().sum() == 0


PORTION_MASKS = [(50, 4, False), (140, 3, False), (140, 128, False), (100, 130, False), (129, 1, False), (300, 500, False), (1, 1, False), (64, 300, False),
                 (4000, 7, False), (128, 0, False), (40, 0, True), (128, 0, True), (200, 0, True), (1, 0, True), (1000, 0, True)]
PORTIONS = [[(0, 300), (0, 1), (0, 51), (0, 700)], [(0, 1100)], [(128, 2), (700, 260), (3, 40), (600, 600)], [(255, 257), (256, 2), (511, 300), (140, 385)],
            [(199, 2), (200, 1), (201, 199), (399, 402)]]


@pytest.mark.parametrize("H,G,D,V,rot", [x for x in SHAPES if x[2] % 8 == 0 and x[3] % 8 == 0 and x[3] <= 128][:5])
@pytest.mark.parametrize("size,keep,chunked", PORTION_MASKS)
@pytest.mark.parametrize("seqs", PORTIONS)
def test_attend_portions_masks_and_gates(H, G, D, V, rot, size, keep, chunked, seqs):
    """Portions of prompts; every row of a sequence is compared, so every 128-row tile meets kept, window and chunk tiles.  The
    kept first keys get large values: a row that misses them is far off."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import KeyMask
    mask = KeyMask(size, keep, chunked)
    s = shape_of(H, G, D, V, rot, mask)
    assert wa.portions_supported(s)
    qs, ks, cu_q, cu_k, want = [], [], [0], [0], []
    fresh = all(start == 0 for start, _ in seqs)
    for b, (start, n) in enumerate(seqs):
        lo, L = mask.first(start), start + n
        q, kv = rnd(n, s.q_width, seed=10 + b, dtype=BF), rnd(L, s.row_width, seed=20 + b, dtype=BF)
        kv[:keep, G * D:] *= 4.0
        for i in (0, n // 2, n - 1):                            # outstanding keys at both sides of the edges
            first = mask.first(start + i)
            for j, f in ((first, 1.5), (first - 1, 3.0), (keep, 3.0)):
                if 0 <= j < L and (j != keep or keep < lo):
                    kv[j, :D] = q[i, :D] * f
        k, v = kv[:, :G * D].double().view(L, G, D), kv[:, G * D:s.kv_width].double().view(L, G, V)
        want.append(O.attend(q.double().view(n, H, D), k, v, s.scale, visible(mask, L, "cuda")[start:]))
        have = list(range(min(keep, lo))) + list(range(lo, L))
        qs.append(q)
        ks.append(kv[have])
        cu_q.append(cu_q[-1] + n)
        cu_k.append(cu_k[-1] + len(have))
    q, rows, want = torch.cat(qs), torch.cat(ks), torch.cat(want)
    for gated in (0, 1, 2):
        gate = {0: None, 1: rnd(cu_q[-1], H + 5, seed=7, dtype=BF)[:, :H], 2: rnd(cu_q[-1], s.out_width + 8, seed=8, dtype=BF)[:, :s.out_width]}[gated]
        out = torch.zeros(cu_q[-1], s.out_width + 8, dtype=BF, device="cuda")
        if fresh:
            wa.attend_portions(torch.cat([q, rows], 1), s, None, i32(*cu_q), i32(*cu_k), max(n for _, n in seqs), out, 1.25, gate)
        else:
            wa.attend_portions(q, s, rows, i32(*cu_q), i32(*cu_k), max(n for _, n in seqs), out, 1.25, gate)
        w = want * 1.25 * (1.0 if gate is None else torch.sigmoid(gate.double()).view(cu_q[-1], H, -1))
        w = w.reshape(cu_q[-1], -1)
        assert rel(out[:, :s.out_width], w) < tol(BF)
        size = w.view(-1, H, V).pow(2).mean(-1).sqrt()
        d = (out[:, :s.out_width].double() - w).view(-1, H, V).pow(2).mean(-1).sqrt() / (size + size.mean())
        assert d.max() < 0.03, (gated, d.max(-1).values.argmax())
        assert out[:, s.out_width:].abs().sum() == 0


# ---------------------------------------------------------------------------------------------- latent attention
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", [dict(heads=2, dim=24, rot=8, vdim=16, rank=48), dict(heads=3, dim=12, rot=6, vdim=20, rank=33),
                                   dict(heads=17, dim=40, rot=16, vdim=24, rank=272)])
def test_latent_prepare_pairs_and_magnitude(dtype, shape):
    from trainscale_b200.ops import latent_attention as L
    r = {"dims": shape["rot"], "base": 700.0, "scaling": O.SCALING}
    s = L.LatentShape(window=8, scale=0.2, rope_base=700.0, pairs=True, magnitude=O.magnitude(r), **shape)
    T, eps = 9, 1e-3
    proj = rnd(T, s.q_width + s.rank + s.rot + 11, seed=1, dtype=dtype)
    src = proj.double().cpu()
    pos, slots = torch.tensor([0, 1, 2, 63, 64, 1000, 5, 400, 17], dtype=torch.int32), torch.tensor([3, 40, 41, 8, 9, 10, 11, 12, 0])
    cache = torch.full((3, 16, s.row_width), 7.0, dtype=dtype).cuda()
    nw = rnd(s.rank, seed=2) + 1.0
    flat = L.prepare(proj, s, nw, eps, O.frequencies(r).float().cuda(), pos.cuda(), slots.cuda(), cache, True)
    at = s.q_width + s.rank
    c = O.rms(src[:, s.q_width:at], eps) * nw.double().cpu()
    kr = O.rotate_pairs(src[:, None, at:at + s.rot], pos, r)[:, 0]
    got = cache.view(-1, s.row_width)[slots.cuda()]
    assert torch.equal(got, flat) and bool((got[:, s.rank + s.rot:] == 0).all())
    loose = 6e-5 if dtype == torch.float32 else 6e-3
    assert rel(got[:, :s.rank], c) < tol(dtype) and rel(got[:, s.rank:s.rank + s.rot], kr) < loose
    q, qs = proj[:, :s.q_width].view(T, s.heads, -1), src[:, :s.q_width].reshape(T, s.heads, -1)
    assert rel(q[..., :s.dim], qs[..., :s.dim]) == 0.0 and rel(q[..., s.dim:], O.rotate_pairs(qs[..., s.dim:], pos, r)) < loose
    assert torch.equal(proj[:, at + s.rot:].double().cpu(), src[:, at + s.rot:])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,K,N", [(1, 3, 24, 40), (9, 2, 64, 128), (40, 5, 12, 33), (100, 2, 96, 64)])
def test_head_products_with_a_gate(dtype, T, H, K, N):
    from trainscale_b200.ops import grouped
    x, w = rnd(T, H, K, seed=1, dtype=dtype), rnd(H, N, K, seed=2, dtype=dtype)
    gate = rnd(T, H * N + 9, seed=3, dtype=dtype)[:, 4:4 + H * N].unflatten(1, (H, N))
    want = torch.einsum("thk,hnk->thn", x.double(), w.double()) * torch.sigmoid(gate.double())
    assert rel(grouped.head_linear(x, w, gate=gate), want) < tol(dtype)


@pytest.mark.parametrize("shape", [dict(heads=2, dim=24, rot=8, vdim=16, rank=48), dict(heads=3, dim=72, rot=40, vdim=80, rank=40),
                                   dict(heads=2, dim=128, rot=64, vdim=128, rank=96)])
@pytest.mark.parametrize("window", [1, 70, 128, 300])
def test_attend_expanded_with_a_gate(shape, window):
    from trainscale_b200.ops import latent_attention as L
    s = L.LatentShape(window=window, scale=0.3, rope_base=1e4, **shape)
    n, past = 400, 90
    lk = n + min(past, window - 1)
    H, D, V = s.heads, s.dim, s.vdim
    proj, kv, rows = rnd(n, s.q_width, seed=1, dtype=BF), rnd(lk, H * (D + V), seed=2, dtype=BF), rnd(lk, s.row_width, seed=3, dtype=BF)
    q, k = proj.double().view(n, H, -1), kv.double()
    kr = rows[:, s.rank:s.rank + s.rot].double()[:, None].expand(lk, H, s.rot)
    want = O.attend(q, torch.cat([k[:, :H * D].view(lk, H, D), kr], -1), k[:, H * D:].view(lk, H, V), s.scale, O.window_mask(lk, window)[lk - n:].cuda())
    for cols in (H, H * V):
        gate = rnd(n, cols + 8 + (-cols) % 8, seed=4, dtype=BF)[:, :cols]
        out = torch.zeros(n, H * V, dtype=BF).cuda()
        L.attend_expanded(proj, kv, rows, s, i32(0, n), i32(0, lk), n, out, gate)
        assert rel(out, (want * torch.sigmoid(gate.double()).view(n, H, -1)).reshape(n, -1)) < 8e-3


# ---------------------------------------------------------------------------------------------- the model
def make_core(cfg, w, dtype, blocks=400, seqs=4, eager=False, block_size=16, budget=4096):
    from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, SchedulerConfig
    from trainscale_b200.models.kabulix import load_model
    ec = EngineConfig(model="custom", tokenizer="byte", device="cuda", dtype=str(dtype)[6:], enforce_eager=eager,
                      scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                      cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=4096))
    return EngineCore(ec, model=load_model(cfg, w, dtype, "cuda"))


class Reference:
    """Logits of whole sequences in fp64, and which positions rounding may route to another expert."""

    def __init__(self, w, cfg):
        self.w, self.cfg = {k: v.double() for k, v in w.items()}, cfg

    def __call__(self, ids):
        return O.logits(self.w, self.cfg, ids)

    def close(self, got, want, dtype, ids, at=None):
        """rms over the vocabulary of the difference (mean taken off), relative to the logits' own spread."""
        d = got.double().cpu() - want
        d = d - d.mean(-1, keepdim=True)
        e = d.pow(2).mean(-1).sqrt() / want.std()
        if dtype == torch.float32:
            return e.max().item() < 5e-5
        turned = O.close_calls(self.w, self.cfg, ids, 0.03)
        clear = torch.ones(len(ids), dtype=torch.bool)
        clear[turned] = False
        if at is not None:
            clear = clear[at]
        return (not clear.any() or e[clear].max().item() < 0.15) and (len(e) < 20 or e.median().item() < 0.03)


def run_portions(core, seq, ids, sizes):
    from trainscale_b200.inference.batch import StepEntry
    out, at, sizes = [], 0, list(sizes)
    while at < len(ids):
        n = min(sizes.pop(0) if sizes else 1, len(ids) - at)
        out.append(core.execute([StepEntry(seq, ids[at:at + n], list(range(n)))]).clone())
        at += n
    return torch.cat(out)


CONFIGS = {
    "mixed": dict(width=128, types=("latent_attention", "attention", "attention_2", "attention"), heads=[6, 4, 8, 6], kv_heads=[2, 4, 2, 1], dim=[32, 64, 24, 40],
                  vdim=[48, 64, 16], window=[40, 129, 17, 70], keep=[2, 5, 1, 130], chunk=[33, 90, 50], rot=[16, 64, 10, 8], lheads=5, ldim=32, lrot=16,
                  lvdim=24, rank=64, lwindow=45, mlps=("moe", "dense", "moe", "moe"), ff=[64, 200], experts=[12, 8, 16, 4], top=[2, 1, 5, 1], groups=[4, 4, 8, 2],
                  keep_groups=[2, 2, 5, 1], expert_ff=[40, 8, 72, 24], shared_ff=[24, 56, 100]),
    "odd": dict(width=90, heads=3, kv_heads=1, dim=18, vdim=10, window=33, keep=7, chunk=29, rot=6, lheads=3, ldim=14, lrot=6, lvdim=9, rank=22, lwindow=31,
                ff=50, expert_ff=11, shared_ff=13, experts=9, top=2, groups=3, keep_groups=1, vocab=301),
    "sinks only": dict(width=64, types=("attention",), heads=2, kv_heads=2, dim=64, window=64, keep=64, rot=64, mlps=(None, "dense")),
    "chunks only": dict(width=64, types=("attention_2", "attention_2"), heads=4, kv_heads=1, dim=64, vdim=128, chunk=[64, 100], mlps=("moe", None)),
    "latent only": dict(width=64, types=("latent_attention",), lheads=2, ldim=64, lrot=64, lvdim=64, rank=128, lwindow=[64], mlps=("moe",)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_whole_prompts_portions_and_decoding(dtype, name):
    cfg = O.make_config(**CONFIGS[name])
    w = O.make_weights(cfg, 3)
    ref, ids = Reference(w, cfg), tokens(333, 1)
    want = ref(ids)
    core = make_core(cfg, w, dtype)
    for i, sizes in enumerate(([333], [100, 2, 2, 31, 64, 1, 1, 5, 90], [300], [2] * 40 + [253], [8, 7, 9, 15, 17, 128, 129])):
        assert ref.close(run_portions(core, i, ids, sizes), want, dtype, ids), sizes
        core.release(i)
    assert core.runner.graph_replays > 30


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_and_long_decoding(dtype):
    """A prompt of several query blocks, and hundreds of tokens decoded one by one past every window and chunk."""
    cfg = O.make_config(width=64, heads=4, kv_heads=2, dim=32, vdim=32, rot=16, window=150, keep=5, chunk=210, ldim=32, lvdim=32, lrot=16,
                        rank=48, lwindow=66, mlps=("dense",))
    w = O.make_weights(cfg, 5)
    ref, ids = Reference(w, cfg), tokens(1100, 2)
    want = ref(ids)
    core = make_core(cfg, w, dtype)
    assert ref.close(run_portions(core, 0, ids, [1100]), want, dtype, ids)
    assert ref.close(run_portions(core, 1, ids, [700, 3]), want, dtype, ids)
    assert ref.close(run_portions(core, 2, ids[:450], [3]), want[:450], dtype, ids[:450])


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_and_reuse(dtype):
    """Unequal requests advance by unequal amounts in one batch, finished ones hand pages on."""
    from trainscale_b200.inference.trace import TraceRunner
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 4)
    ref = Reference(w, cfg)
    core = make_core(cfg, w, dtype, blocks=40, seqs=3)
    reqs = {f"r{i}": tokens(n, 50 + i) for i, n in enumerate([150, 3, 97, 1, 210, 45, 64, 2])}
    waiting, live, at, step = list(reqs), [], {}, 0
    runner, got = TraceRunner(core), {r: [] for r in reqs}
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
        entries, end = [], []
        for j, r in enumerate(live):
            lo = at.get(r, 0)
            n = min([1, 40, 2, 17, 1, 8, 64][(step + j) % 7], len(reqs[r]) - lo)
            if (step + 2 * j) % 6 == 5:
                continue
            entries.append({"id": r, "tokens": reqs[r][lo:lo + n], "want": list(range(n))})
            at[r] = lo + n
            if at[r] == len(reqs[r]):
                end.append(r)
        logits = runner.run({"step": step, "entries": entries, "end": end})
        row = 0
        for e in entries:
            got[e["id"]].append(logits[row:row + len(e["want"])].clone())
            row += len(e["want"])
        live = [r for r in live if r not in end]
        step += 1
    for r, ids in reqs.items():
        assert ref.close(torch.cat(got[r]), ref(ids), dtype, ids), r
    assert core.cache.alloc.num_free == 40


def test_wide_decode_batch():
    """More rows than the few-row products take, odd batch sizes, captured and not."""
    from trainscale_b200.inference.batch import StepEntry
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 6)
    ref = Reference(w, cfg)
    reqs = [tokens(5 + (7 * i) % 60, 100 + i) for i in range(45)]
    want = [ref(r)[-1] for r in reqs]
    for eager in (True, False):
        core = make_core(cfg, w, BF, seqs=45, eager=eager)
        for i, r in enumerate(reqs):
            core.execute([StepEntry(i, r[:-1], [])])
        got = core.execute([StepEntry(i, [r[-1]]) for i, r in enumerate(reqs)])
        for i, r in enumerate(reqs):
            assert ref.close(got[i:i + 1], want[i][None], BF, r, [len(r) - 1]), (eager, i)


def test_generation_fp32_matches_oracle():
    """Greedy tokens of the engine's own entry point, with chunked prefill and preemption."""
    from trainscale_b200.inference import GenerationParams, SOTAInferenceEngine
    cfg = O.make_config(width=64, window=20, chunk=25, lwindow=18)
    w = O.make_weights(cfg, 7, sharp=1.5)
    prompts = [tokens(n, n) for n in (40, 3, 77, 18)]
    want = [O.greedy({k: v.double() for k, v in w.items()}, cfg, p, 12) for p in prompts]
    for kw in (dict(), dict(budget=16), dict(blocks=10, budget=32)):
        core = make_core(cfg, w, torch.float32, **kw)
        eng = SOTAInferenceEngine.__new__(SOTAInferenceEngine)
        eng.config, eng.core, eng.draft_model = core.config, core, None
        res = eng.generate(prompts, GenerationParams(max_tokens=12, temperature=0.0, ignore_eos=True)).unwrap()
        assert [r.token_ids for r in res] == want, kw


def test_forward_equals_engine_and_kernels_report_no_error():
    from trainscale_b200.ops import _lib
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 8)
    core = make_core(cfg, w, BF)
    ids = tokens(70, 3)
    a = core.model(torch.tensor([ids, ids[::-1]]))
    b = run_portions(core, 0, ids, [70])
    d = (a[0] - b).pow(2).mean(-1).sqrt() / b.std()
    assert d.median() < 0.02 and math.isfinite(a.sum().item())
    _lib.raise_on_loaded_device_error()
