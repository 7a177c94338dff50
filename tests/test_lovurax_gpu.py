"""Lovurax kernels and the model on the GPU against plain fp64 PyTorch (lovurax_oracle.py and the formulas below)."""
import math

import pytest
import torch
import torch.nn.functional as F

import lovurax_oracle as O

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
@pytest.mark.parametrize("base", [0.0, 1.0])
@pytest.mark.parametrize("T,W", [(5, 64), (3, 66), (7, 2048), (2, 6144), (4, 1030), (300, 256), (1, 1), (3, 8)])
def test_boundary_with_a_gate_per_element(dtype, base, T, W):
    from trainscale_b200.ops import stream
    x, w, b = rnd(T, W, seed=1), rnd(W, seed=3, scale=0.3) + 1, rnd(W, seed=5)
    y = rnd(T, W + (8 if W % 4 == 0 else 3), seed=2, dtype=dtype, scale=3.0)[:, :W]
    z = rnd(T, W + 24, seed=4, dtype=dtype, scale=2.0)[:, 16:16 + W]
    want = x.double() + y.double() * torch.sigmoid(z.double() + b.double())
    h = O.rms(want, 1e-5) * (base + w.double())
    gate = stream.ElementGate(z, b)
    xo, ho = stream.prenorm(x, y, gate, None, w, 1e-5, dtype, base)
    assert rel(xo, want) < 1e-6 and rel(ho, h) < tol(dtype)
    rows = torch.randperm(T, generator=torch.Generator().manual_seed(6))[:max(1, T // 2)].int().cuda()
    assert rel(stream.prenorm_final(x, y, gate, None, w, 1e-5, rows, dtype, base), h[rows.long()]) < tol(dtype)
    table, tok = rnd(50, W, seed=7, dtype=dtype), torch.randint(0, 50, (T,), generator=torch.Generator().manual_seed(8)).cuda()
    x0, h0 = stream.prenorm_embed(tok, table, w, 1e-5, base)
    assert torch.equal(x0, table[tok].float()) and rel(h0, O.rms(x0.double(), 1e-5) * (base + w.double())) < tol(dtype)


# ---------------------------------------------------------------------------------------------- products
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K,cols", [(3, 40, 64, 32), (20, 96, 128, 96), (70, 300, 64, 256), (600, 512, 256, 64), (2500, 1032, 192, 1024),
                                        (5, 41, 21, 32), (1, 64, 64, 0), (33, 64, 64, 32), (700, 520, 136, 512)])
def test_activation_of_leading_columns(dtype, M, N, K, cols):
    """xIELU of the first columns, the others as they are; a constant factor of all."""
    from trainscale_b200.ops import gemm, grouped
    x, w = rnd(M, K, seed=1, dtype=dtype), rnd(N, K, seed=2, dtype=dtype, scale=1.5 / math.sqrt(K))
    z = x.double() @ w.double().t()
    p, q = torch.tensor([0.7, -0.4], dtype=torch.float64)
    a, b = F.softplus(p).item(), 0.5 + F.softplus(q).item()
    want = torch.cat([O.xielu(z[:, :cols].cpu(), p, q), z[:, cols:].cpu()], -1)
    got = gemm.serve_linear(x, w, act=grouped.ACT_XIELU, cap=a, second=b, act_cols=cols)
    assert rel(got, want) < tol(dtype)
    if cols not in (0, N):
        assert rel(got[:, :cols], want[:, :cols]) < tol(dtype) and rel(got[:, cols:], want[:, cols:]) < tol(dtype)
    assert rel(gemm.serve_linear(x, w, torch.float32, act=grouped.ACT_XIELU, cap=a, second=b), O.xielu(z.cpu(), p, q)) < 1e-5
    assert rel(gemm.serve_linear(x, w, torch.float32, act=grouped.ACT_SCALE, cap=-0.37), -0.37 * z) < 4e-6


@pytest.mark.parametrize("M", [4, 400])
@pytest.mark.parametrize("scale", [1e-6, 1e-3, 0.05, 1.0, 30.0])
def test_xielu_keeps_its_digits_near_zero_and_far_out(M, scale):
    """The exponential's difference must not cancel, nor the square or the exponential overflow.  (The GEMM's epilogue is made for
    results that are rounded to 16 bits.)"""
    from trainscale_b200.ops import gemm, grouped
    x, w = torch.eye(64, dtype=BF).repeat(M // 4, 1)[:M * 16].cuda(), rnd(64, 64, seed=1, dtype=BF, scale=scale)
    z = x.double() @ w.double().t()
    got = gemm.serve_linear(x, w, torch.float32, act=grouped.ACT_XIELU, cap=1.3, second=0.9).double()
    n = z.clamp(max=0.0)
    want = 1.3 * z.clamp(min=0.0) ** 2 + 0.9 * (torch.expm1(n) - n) + z / 2
    assert ((got - want).abs() / (want.abs() + z.abs() / 2).clamp(min=1e-30)).max() < (3e-6 if M == 4 else 1e-4)     # left of zero the terms may cancel


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,K,N", [(1, 3, 24, 40), (9, 2, 64, 128), (40, 5, 12, 33), (100, 2, 96, 64)])
def test_head_products_with_a_gate_per_head(dtype, T, H, K, N):
    from trainscale_b200.ops import grouped
    x, w = rnd(T, H, K, seed=1, dtype=dtype), rnd(H, N, K, seed=2, dtype=dtype)
    gate = rnd(T, H + 9, seed=3, dtype=dtype)[:, 4:4 + H]
    want = torch.einsum("thk,hnk->thn", x.double(), w.double()) * torch.sigmoid(gate.double())[:, :, None]
    assert rel(grouped.head_linear(x, w, gate=gate[:, :, None].expand(-1, -1, N)), want) < tol(dtype)


# ---------------------------------------------------------------------------------------------- attention
SHAPES = [(5, 1, 96, 96), (8, 2, 128, 128), (4, 4, 64, 64), (5, 5, 40, 72), (24, 1, 80, 48), (3, 1, 20, 12), (4, 2, 18, 30), (2, 1, 256, 128),
          (2, 2, 200, 256), (1, 1, 8, 8)]      # H, G, dim, vdim


def shape_of(H, G, D, V, mask, **kw):
    from trainscale_b200.ops.window_attention import WindowShape
    return WindowShape(H, G, D, V, 0, mask.size, D ** -0.5 * 1.3, mask.keep, mask.chunked, **kw)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", SHAPES)
@pytest.mark.parametrize("every,coef,normed", [(64, 0.4, True), (1, 0.1, True), (100000, 0.7, True), (7, -0.2, False)])
def test_prepare_with_a_query_temperature(dtype, H, G, D, V, every, coef, normed):
    """Positions on both sides of the places where the factor grows; keys and values stay without it."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import KeyMask
    s = shape_of(H, G, D, V, KeyMask(9), sigmoid=True, temperature=(coef, every))
    pos = [0, 1, 5, 6, 7, 62, 63, 64, 126, 127, 128, 4000, 99998, 99999, 100000, 199999]
    T = len(pos)
    proj = rnd(T, s.q_width + s.kv_width + 8 + (-(s.q_width + s.kv_width)) % 8, seed=1, dtype=dtype)
    before = proj.clone()
    qn, kn = (rnd(D, seed=2), rnd(D, seed=3)) if normed else (None, None)
    cache = torch.zeros(4, 8, s.row_width, dtype=dtype, device="cuda")
    slots = torch.randperm(32, generator=torch.Generator().manual_seed(5))[:T].cuda()
    wa.prepare(proj, s, qn, kn, 1e-5, None, slots, cache, pos=i32(*pos))
    x, qw, kw = before.double().cpu(), s.q_width, G * D
    f = torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in pos], dtype=torch.float64)[:, None, None]

    def changed(y, w):
        return O.norm(y, w.double().cpu(), 1e-5) if normed else y

    assert rel(proj[:, :qw], (changed(x[:, :qw].reshape(T, H, D), qn) * f).reshape(T, -1)) < tol(dtype)
    assert rel(proj[:, qw:qw + kw], changed(x[:, qw:qw + kw].reshape(T, G, D), kn).reshape(T, -1)) < tol(dtype)
    assert torch.equal(proj[:, qw + kw:], before[:, qw + kw:])
    rows = cache.view(-1, s.row_width)[slots]
    assert torch.equal(rows[:, :s.kv_width], proj[:, qw:qw + s.kv_width])


def attend(q, k, v, scale, distance, visible, slopes, add, sigmoid):
    """q [Tq, H, D], k [Tk, G, D], v [Tk, G, V], distance and visible [Tq, Tk]."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        s = q[:, h] @ k[:, h // (H // G)].t() * scale
        if slopes is not None:
            s = s - slopes[h].double() * distance
        if add is not None:
            s = s + add[h].double()
        w = torch.sigmoid(s).masked_fill(~visible, 0.0) if sigmoid else torch.softmax(s.masked_fill(~visible, -math.inf), -1)
        out.append(w @ v[:, h // (H // G)])
    return torch.stack(out, 1)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", SHAPES)
@pytest.mark.parametrize("sigmoid,sloped,added", [(True, True, True), (True, False, True), (True, True, False), (False, True, True), (True, False, False)])
@pytest.mark.parametrize("size,keep,chunked", [(1 << 30, 0, False), (50, 4, False), (40, 0, True)])
def test_attend_rows_with_biased_scores(dtype, H, G, D, V, sigmoid, sloped, added, size, keep, chunked):
    """Single query rows against scattered pages, long enough for several splits.  The first key of every row stands out, whatever
    its distance takes off."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import KeyMask
    mask, bs = KeyMask(size, keep, chunked), 16
    s = shape_of(H, G, D, V, mask, sigmoid=sigmoid)
    lens = [1, 2, 15, 16, 17, 129, 700, 2500]
    n, nb = len(lens), 2500 // bs + 50
    perm = torch.randperm(n * nb + 3, generator=torch.Generator().manual_seed(1))[:n * nb].view(n, nb).int()
    cache = rnd(n * nb + 3, bs, s.row_width, seed=2, dtype=dtype)
    q = rnd(n, s.q_width + 16 + (-s.q_width) % 8, seed=3, dtype=dtype)
    flat = cache.view(-1, s.row_width)
    slots = [torch.tensor([int(perm[b, j // bs]) * bs + j % bs for j in range(L)]).cuda() for b, L in enumerate(lens)]
    slopes = wa.distance_slopes(H).cuda() * 0.05 if sloped else None
    add = rnd(H, seed=9) - 6.0 if added else None
    for b, L in enumerate(lens):
        far = 0.05 * 2.0 ** (-8.0 / H) * L if sloped else 0.0
        flat[slots[b][0], :D] = q[b, :D] * ((far + 8) / (s.scale * q[b, :D].float().pow(2).sum())).to(dtype)
    gate = rnd(n, s.out_width + 8, seed=8, dtype=dtype)[:, :s.out_width]
    out = torch.zeros(n, s.out_width + 8, dtype=dtype, device="cuda")
    wa.attend_rows(q, s, cache, perm.cuda(), torch.arange(n, dtype=torch.int32, device="cuda"), i32(*lens), max(lens), out[:, :s.out_width], 0.75, gate,
                   wa.ScoreBias(slopes, add))
    for b, L in enumerate(lens):
        j = torch.tensor(mask.positions(L - 1)).cuda()
        rows = flat[slots[b][j]].double()
        k, v = rows[:, :G * D].view(-1, G, D), rows[:, G * D:s.kv_width].view(-1, G, V)
        want = attend(q[b:b + 1, :s.q_width].double().view(1, H, D), k, v, s.scale, (L - 1 - j)[None].double(),
                      torch.ones(1, len(j), dtype=torch.bool, device="cuda"), slopes, add, sigmoid)
        want = want * 0.75 * torch.sigmoid(gate[b].double()).view(1, H, V)
        assert rel(out[b, :s.out_width], want.reshape(-1)) < tol(dtype, 1.5), (b, L)
    assert out[:, s.out_width:].abs().sum() == 0


PORTIONS = [[(0, 300), (0, 1), (0, 51), (0, 700)], [(0, 1100)], [(128, 2), (700, 260), (3, 40), (600, 600)], [(255, 257), (256, 2), (511, 300), (140, 385)],
            [(199, 2), (200, 1), (201, 199), (399, 402)]]


@pytest.mark.parametrize("H,G,D,V", [x for x in SHAPES if x[2] % 8 == 0 and x[3] % 8 == 0 and x[3] <= 128])
@pytest.mark.parametrize("sloped,added", [(True, True), (False, False)])
@pytest.mark.parametrize("size,keep,chunked", [(1 << 30, 0, False), (140, 3, False), (129, 130, False), (200, 0, True)])
@pytest.mark.parametrize("seqs", PORTIONS)
def test_attend_portions_with_sigmoid_weights(H, G, D, V, sloped, added, size, keep, chunked, seqs):
    """Every row of every portion, so every tile's border and diagonal.  Weights are small except at each sequence's first key and
    at the edges: a row that misses one of them, or sees the key behind it, is far off."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import KeyMask
    mask = KeyMask(size, keep, chunked)
    s = shape_of(H, G, D, V, mask, sigmoid=True)
    assert wa.portions_supported(s)
    slopes = wa.distance_slopes(H).cuda() * 0.02 if sloped else None
    add = rnd(H, seed=9) - 6.0 if added else None
    qs, ks, cu_q, cu_k, want = [], [], [0], [0], []
    fresh = all(start == 0 for start, _ in seqs)
    for b, (start, n) in enumerate(seqs):
        lo, L = mask.first(start), start + n
        q, kv = rnd(n, s.q_width, seed=10 + b, dtype=BF), rnd(L, s.row_width, seed=20 + b, dtype=BF)
        for i in (0, n // 2, n - 1):
            p = start + i
            for j in {0, keep, mask.first(p), mask.first(p) - 1, p, p + 1, max(0, p - 127), max(0, p - 128)}:
                if 0 <= j < L:
                    f = (0.02 * 2.0 ** (-8.0 / H) * abs(p - j) if sloped else 0.0) + 8
                    kv[j, :D] = q[i, :D] * (f / (s.scale * q[i, :D].float().pow(2).sum())).to(BF)
        k, v = kv[:, :G * D].double().view(L, G, D), kv[:, G * D:s.kv_width].double().view(L, G, V)
        i, j = torch.arange(start, L, device="cuda")[:, None], torch.arange(L, device="cuda")[None]
        vis = torch.zeros(n, L, dtype=torch.bool)
        for r in range(n):
            vis[r, mask.positions(start + r)] = True
        want.append(attend(q.double().view(n, H, D), k, v, s.scale, (i - j).double(), vis.cuda(), slopes, add, True))
        have = list(range(min(keep, lo))) + list(range(lo, L))
        qs.append(q)
        ks.append(kv[have])
        cu_q.append(cu_q[-1] + n)
        cu_k.append(cu_k[-1] + len(have))
    if sloped and keep and not fresh:
        return                              # kept keys stand right before the window: their distance is not that of the rows
    q, rows, want = torch.cat(qs), torch.cat(ks), torch.cat(want)
    gate = rnd(cu_q[-1], s.out_width + 8, seed=8, dtype=BF)[:, :s.out_width]
    out = torch.zeros(cu_q[-1], s.out_width + 8, dtype=BF, device="cuda")
    if fresh:
        wa.attend_portions(torch.cat([q, rows], 1), s, None, i32(*cu_q), i32(*cu_k), max(n for _, n in seqs), out, 1.25, gate, wa.ScoreBias(slopes, add))
    else:
        wa.attend_portions(q, s, rows, i32(*cu_q), i32(*cu_k), max(n for _, n in seqs), out, 1.25, gate, wa.ScoreBias(slopes, add))
    w = (want * 1.25 * torch.sigmoid(gate.double()).view(cu_q[-1], H, V)).reshape(cu_q[-1], -1)
    assert rel(out[:, :s.out_width], w) < tol(BF)
    size = w.view(-1, H, V).pow(2).mean(-1).sqrt()
    d = (out[:, :s.out_width].double() - w).view(-1, H, V).pow(2).mean(-1).sqrt() / (size + size.mean())
    assert d.max() < 0.03, d.max(-1).values.argmax()
    assert out[:, s.out_width:].abs().sum() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V", [(8, 2, 64, 64), (5, 1, 96, 40), (1, 1, 32, 128), (24, 3, 16, 16)])
@pytest.mark.parametrize("shift", [-6.0, 30.0])
def test_sigmoid_weights_that_fade_with_the_distance(dtype, H, G, D, V, shift):
    """With the scores' bound known, far keys are left out: the result stays that of all keys.  One key stands out as far as the
    bound allows, just where its weight is still large."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import UNBOUNDED
    n, bs = 1500, 16
    s = wa.WindowShape(H, G, D, V, 0, UNBOUNDED, D ** -0.5, sigmoid=True)
    q, kv = rnd(n, s.q_width, seed=1, dtype=dtype), rnd(n + 4, s.row_width, seed=2, dtype=dtype)
    slopes, add = wa.distance_slopes(H).cuda(), rnd(H, seed=3) + shift
    for h in range(H):
        reach = min(n - 1, int((30.0 + add[h].item()) / slopes[h].item()))          # a score of 30 there has a weight of about one half
        if reach >= 0:
            g = h // (H // G)
            u = q[n - 1, h * D:(h + 1) * D].float()
            kv[n - 1 - reach, g * D:(g + 1) * D] = (u * (30.0 / (s.scale * u.pow(2).sum()))).to(dtype)
    k, v = kv[:n, :G * D].double().view(n, G, D), kv[:n, G * D:s.kv_width].double().view(n, G, V)
    rows = [n - 1, n - 2, 700, 100, 1, 0]
    i, j = torch.tensor(rows, device="cuda")[:, None], torch.arange(n, device="cuda")[None]
    products = torch.stack([q[:, h * D:(h + 1) * D].double() @ k[:, h // (H // G)].t() for h in range(H)]).max().item() * s.scale
    bias = wa.ScoreBias(slopes, add, products * 1.001)
    assert H == 1 or min(wa.sigmoid_reach(bias.limit, a, b) for a, b in zip(add.tolist(), slopes.tolist())) < 700
    want = attend(q[rows].double().view(len(rows), H, D), k, v, s.scale, (i - j).double(), j <= i, slopes, add, True).reshape(len(rows), -1)
    out = torch.zeros(len(rows), s.out_width, dtype=dtype, device="cuda")
    table = torch.arange((n + 4) // bs, dtype=torch.int32, device="cuda")[None]
    wa.attend_rows(q[rows].contiguous(), s, kv.view(-1, bs, s.row_width), table, i32(*[0] * len(rows)), i32(*[r + 1 for r in rows]), n, out, bias=bias)
    assert rel(out, want) < tol(dtype, 1.5) and all(rel(out[x], want[x]) < tol(dtype, 2.0) for x in range(len(rows)))
    if dtype == BF:
        whole = torch.zeros(n, s.out_width, dtype=BF, device="cuda")
        wa.attend_portions(torch.cat([q, kv[:n]], 1), s, None, i32(0, n), i32(0, n), n, whole, bias=bias)
        assert rel(whole[rows], want) < tol(BF)
        wa.attend_portions(q[900:].contiguous(), s, kv[:n].contiguous(), i32(0, n - 900), i32(0, n), n - 900, whole, bias=bias)
        assert rel(whole[[n - 901, n - 902]], want[:2]) < tol(BF)


def test_sigmoid_weights_far_below_and_above_one():
    """Scores of hundreds either way: weights of zero and one, no overflow where two of them share a reciprocal."""
    from trainscale_b200.ops import window_attention as wa
    from trainscale_b200.ops.masks import UNBOUNDED
    s = wa.WindowShape(2, 1, 64, 64, 0, UNBOUNDED, 1.0, sigmoid=True)
    n = 300
    q, kv = torch.zeros(n, s.q_width, dtype=BF, device="cuda"), rnd(n, s.row_width, seed=1, dtype=BF)
    q[:, 0] = q[:, 64] = 20.0
    kv[:, :64] = 0
    kv[:, 0] = torch.tensor([1000.0, -1000.0, 30.0, -30.0, 0.0, -4.0, -5.0])[torch.arange(n) % 7].cuda().to(BF)
    want = attend(q.double().view(n, 2, 64), kv[:, None, :64].double(), kv[:, None, 64:128].double(), 1.0, torch.zeros(n, n).cuda(),
                  torch.tril(torch.ones(n, n, dtype=torch.bool)).cuda(), None, None, True).reshape(n, -1)
    out = torch.zeros(n, s.out_width, dtype=BF, device="cuda")
    wa.attend_portions(torch.cat([q, kv], 1), s, None, i32(0, n), i32(0, n), n, out)
    assert rel(out, want) < tol(BF)
    cache = torch.cat([kv, kv[:20]]).view(20, 16, -1)
    wa.attend_rows(q[-1:], s, cache, torch.arange(20, dtype=torch.int32, device="cuda")[None], i32(0), i32(n), n, out[:1])
    assert rel(out[0], want[-1]) < tol(BF)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,dim,vdim,rank", [(3, 24, 16, 48), (2, 12, 20, 33), (5, 64, 72, 80), (17, 40, 24, 272)])
def test_latent_attention_without_positions(dtype, heads, dim, vdim, rank):
    """No rotated part and no window: cache rows, the latent form of single rows and, where it runs, the expanded form of portions."""
    from trainscale_b200.ops import latent_attention as L
    from trainscale_b200.ops.masks import UNBOUNDED
    s = L.LatentShape(heads, dim, 0, vdim, rank, UNBOUNDED, 0.4)
    n, bs, eps = 300, 16, 1e-3
    pad = 8 + (-(s.q_width + rank)) % 8
    proj, nw = rnd(n, s.q_width + rank + pad, seed=1, dtype=dtype), rnd(rank, seed=2) * 0.2 + 1
    before, slots = proj.clone(), torch.randperm(20 * bs, generator=torch.Generator().manual_seed(3))[:n]
    table = torch.arange(20, dtype=torch.int32)[None].cuda()
    cache = torch.full((20, bs, s.row_width), 7.0, dtype=dtype, device="cuda")
    freq = torch.empty(0, dtype=torch.float32, device="cuda")
    flat = L.prepare(proj, s, nw, eps, freq, torch.arange(n, dtype=torch.int32, device="cuda"), slots.cuda(), cache, True)
    c = O.norm(before[:, s.q_width:s.q_width + rank].double().cpu(), nw.double().cpu(), eps)
    assert torch.equal(proj, before) and rel(flat[:, :rank], c) < tol(dtype) and flat[:, rank:].abs().sum() == 0
    assert torch.equal(cache.view(-1, s.row_width)[slots.cuda()], flat)
    # single rows see the cache in page order
    cache.view(-1, s.row_width)[:n] = flat
    w = rnd(heads * (dim + vdim), rank, seed=4, dtype=dtype, scale=rank ** -0.5)
    uk, uv = (z.double().cpu() for z in (w[:heads * dim].view(heads, dim, rank), w[heads * dim:].view(heads, vdim, rank)))
    cc, q = flat[:, :rank].double().cpu(), before[:, :s.q_width].double().cpu().view(n, heads, dim)
    q_lat = torch.einsum("thd,hdr->thr", q, uk)
    sc = torch.einsum("thr,jr->htj", q_lat, cc) * s.scale
    w8 = torch.softmax(sc.masked_fill(torch.arange(n)[:, None] < torch.arange(n), -math.inf), -1)
    rows = torch.tensor([0, 1, 15, 16, 128, n - 1])
    lat = L.attend_latent(q_lat.to(dtype).cuda()[rows.cuda()].contiguous(), proj[rows.cuda()], s, cache, table, i32(*[0] * len(rows)),
                          (rows + 1).int().cuda(), n)
    assert rel(lat, torch.einsum("htj,jr->thr", w8, cc)[rows]) < tol(dtype, 1.5)
    if dtype == BF and L.expanded_supported(s):
        kv = (cc @ w.double().cpu().t()).to(dtype).cuda()
        gate = rnd(n, heads + 5, seed=5, dtype=dtype)[:, :heads]
        out = torch.zeros(n, heads * vdim, dtype=dtype, device="cuda")
        L.attend_expanded(proj, kv, flat, s, i32(0, n), i32(0, n), n, out, gate)
        want = torch.einsum("htj,jr,hvr->thv", w8, cc, uv) * torch.sigmoid(gate.double().cpu())[:, :, None]
        assert rel(out, want.reshape(n, -1)) < 8e-3


# ---------------------------------------------------------------------------------------------- retention
RETENTION = [(5, 32, 64, 32), (2, 64, 64, 16), (3, 128, 256, 128), (2, 128, 128, 64), (5, 8, 8, 4), (2, 24, 40, 16), (3, 20, 36, 6), (1, 17, 9, 2),
             (2, 256, 128, 64), (2, 96, 200, 96), (2, 64, 512, 64), (2, 40, 72, 0), (1, 72, 320, 48), (3, 80, 16, 10)]      # H, D, V, rotated
DECAYS = (0.97, 0.9995, 0.5, 0.995, 1.0)


def retention_case(H, D, V, rot, T, dtype, seed=0, first=0):
    from trainscale_b200.ops.recurrent import RetentionShape
    s = RetentionShape(H, D, V, rot, tuple(DECAYS[h % 5] for h in range(H)))
    proj = rnd(T, -(-s.proj_width // 8) * 8 + 8, seed=seed + 1, dtype=dtype)
    a = (torch.arange(T) + first).double()[:, None] * torch.tensor([100.0 ** (-2.0 * i / max(rot, 1)) for i in range(rot // 2)], dtype=torch.float64)
    return s, proj, torch.cat([a.cos(), a.sin()], -1).float().cuda(), rnd(30, s.state_width, seed=seed + 2, scale=0.5)


def retention_oracle(s, x, cs, state, eps):
    """One sequence: x [T, proj_width] fp64, cosines and sines [T, rot], state row or None -> gated result, matrices."""
    T, H, D, V, half = x.shape[0], s.heads, s.dim, s.vdim, s.rot // 2
    c, n = cs[:, None, :half], cs[:, None, half:]

    def turned(y):
        y = y.reshape(T, H, D)
        u, v = y[..., :half], y[..., half:s.rot]
        return torch.cat([u * c - v * n, v * c + u * n, y[..., s.rot:]], -1)

    kw = H * D
    q, k, v = turned(x[:, :kw]), turned(x[:, kw:2 * kw]) * D ** -0.5, x[:, 2 * kw:2 * kw + H * V].reshape(T, H, V)
    S = torch.zeros(H, D, V, dtype=torch.float64) if state is None else state[:H * D * V].view(H, D, V).clone()
    g, out = torch.tensor(s.decay, dtype=torch.float32).double()[:, None, None], []
    for t in range(T):
        S = g * S + k[t, :, :, None] * v[t, :, None]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    o = O.rms(torch.stack(out), eps).reshape(T, -1) * O.silu(x[:, 2 * kw + H * V:s.proj_width])
    return o, S


PREV = [3, -1, 7, 5, -1]


def _portions(lens):
    from trainscale_b200.inference.batch import Portions
    at = [0]
    for n in lens:
        at.append(at[-1] + n)
    return Portions(at, i32(*at))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V,rot", RETENTION)
@pytest.mark.parametrize("lens", [[5, 9, 2, 33, 8], [300], [128, 2, 129, 127, 41], [2, 256, 8, 7, 255]])
def test_retention_portions(dtype, H, D, V, rot, lens):
    """Portions that continue a state or start from zero, some of whole blocks and chunks, behind single rows; results and the
    states they leave, the other state rows untouched."""
    from trainscale_b200.ops import recurrent
    from trainscale_b200.ops.stream import StreamRows
    T, ns, eps = sum(lens), 3, 1e-5
    s, proj, cs, state = retention_case(H, D, V, rot, T + ns, dtype)
    prev, nxt = [-1] * ns, [-1] * ns
    for b, n in enumerate(lens):
        prev += [PREV[b]] + [-2] * (n - 1)
        nxt += [-1] * (n - 1) + [20 + b]
    out = torch.zeros(T + ns, -(-s.out_width // 8) * 8 + 8, dtype=dtype, device="cuda")
    before, powers = state.clone(), s.powers().cuda()
    recurrent.retention(proj[:, :s.proj_width], s, powers, eps, cs, StreamRows(i32(*prev), i32(*nxt)), state, ns, _portions(lens), out[:, :s.out_width])
    at = ns
    for b, n in enumerate(lens):
        o, S = retention_oracle(s, proj[at:at + n, :s.proj_width].double().cpu(), cs[at:at + n].double().cpu(),
                                before[PREV[b]].double().cpu() if PREV[b] >= 0 else None, eps)
        assert rel(out[at:at + n, :s.out_width], o) < tol(dtype, 2.0), (b, n)
        assert rel(state[20 + b, :S.numel()], S.reshape(-1)) < 6e-6, (b, n)
        at += n
    assert torch.equal(state[:20], before[:20]) and torch.equal(state[20 + len(lens):], before[20 + len(lens):]) and out[:, s.out_width:].abs().sum() == 0


@pytest.mark.parametrize("D,V", [(128, 256), (64, 64), (48, 64), (128, 128)])
def test_retention_chunks_keep_fp32_accuracy(D, V):
    """What the chunks add up, before it is rounded to bf16: against fp64, with large queries and keys, far below bf16 rounding."""
    from trainscale_b200.ops import recurrent
    from trainscale_b200.ops.stream import StreamRows
    n, H = 700, 5
    s, proj, cs, state = retention_case(H, D, V, D, n, BF, seed=9)
    proj[:, 2 * s.qk_width + s.out_width:] = 20.0            # silu(20) = 20: the gate passes the norm's result
    out = torch.zeros(n, s.out_width, dtype=BF, device="cuda")
    tail = StreamRows(i32(*[4] + [-2] * (n - 1)), i32(*[-1] * (n - 1) + [21]))
    recurrent.retention_chunks(proj, s, s.powers().cuda(), 1e-6, cs, tail, state, _portions([n]), out)
    o, S = retention_oracle(s, proj[:, :s.proj_width].double().cpu(), cs.double().cpu(), state[4].double().cpu(), 1e-6)
    assert rel(state[21, :S.numel()], S.reshape(-1)) < 2e-6
    # a bf16 result that is the fp64 one rounded, but for ties
    assert (out.cpu() != o.to(BF)).float().mean() < 2e-3 and rel(out, o) < 2.5e-3


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,V,rot", RETENTION)
def test_retention_steps_equal_a_portion(dtype, H, D, V, rot):
    """Token-by-token decoding of two sequences (state rows taking turns) gives what one portion gives."""
    from trainscale_b200.ops import recurrent
    from trainscale_b200.ops.stream import StreamRows
    n, eps = 21, 1e-5
    s, proj, cs, state = retention_case(H, D, V, rot, 2 * n, dtype, seed=40)
    first, powers = state[4].double().cpu(), s.powers().cuda()
    outs = torch.zeros(2 * n, s.out_width, dtype=dtype, device="cuda")
    for t in range(n):
        prev = i32(10 + (t & 1), 12 + (t & 1)) if t else i32(-1, 4)
        rows = StreamRows(prev, i32(10 + ((t + 1) & 1), 12 + ((t + 1) & 1)))
        o = torch.empty(2, s.out_width, dtype=dtype, device="cuda")
        recurrent.retention(proj[[t, n + t]], s, powers, eps, cs[[t, n + t]].contiguous(), rows, state, 2, None, o)
        outs[t], outs[n + t] = o[0], o[1]
    for b, st in ((0, None), (1, first)):
        o, S = retention_oracle(s, proj[b * n:(b + 1) * n, :s.proj_width].double().cpu(), cs[b * n:(b + 1) * n].double().cpu(), st, eps)
        assert rel(outs[b * n:(b + 1) * n], o) < tol(dtype, 2.0)
        assert rel(state[10 + 2 * b + (n & 1), :S.numel()], S.reshape(-1)) < 6e-6


# ---------------------------------------------------------------------------------------------- the model
def make_core(cfg, w, dtype, blocks=400, seqs=4, eager=False, block_size=16, budget=4096):
    from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, SchedulerConfig
    from trainscale_b200.models.lovurax import load_model
    ec = EngineConfig(model="custom", tokenizer="byte", device="cuda", dtype=str(dtype)[6:], enforce_eager=eager,
                      scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                      cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=4096))
    return EngineCore(ec, model=load_model(cfg, w, dtype, "cuda"))


def oracle(w, cfg, ids):
    return O.logits({k: v.double() for k, v in w.items()}, cfg, ids)


def close(got, want, dtype):
    """rms over the vocabulary of the difference (mean taken off), relative to the logits' own spread."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / want.std()
    return e.max().item() < (5e-5 if dtype == torch.float32 else 0.12) and (dtype == torch.float32 or len(e) < 20 or e.median().item() < 0.03)


def run_portions(core, seq, ids, sizes):
    from trainscale_b200.inference.batch import StepEntry
    out, at, sizes = [], 0, list(sizes)
    while at < len(ids):
        n = min(sizes.pop(0) if sizes else 1, len(ids) - at)
        out.append(core.execute([StepEntry(seq, ids[at:at + n], list(range(n)))]).clone())
        at += n
    return torch.cat(out)


CONFIGS = {
    "mixed": dict(width=136, types=("attention", "retention", "latent_attention", "retention", "attention"), heads=[6, 4, 8, 6, 2], kv_heads=[2, 4, 2, 1, 1],
                  dim=[32, 64, 24, 40, 56], vdim=[48, 64, 16, 8, 72], temp=[0.5, 0.1, 0.3], every=[64, 10, 33], rheads=[3, 5, 1, 2], rdim=[24, 32, 8, 64],
                  rvdim=[72, 16, 8, 80], rot=[16, 8, 4, 64], base=[1000.0, 30.0, 5e5], decay=[(0.9, 0.99, 0.6), (0.999, 0.95), (0.8,)], lheads=5, ldim=48, lvdim=24,
                  rank=72, mlps=(1, 1, 0, 1), ff=[200, 33, 64], logit_scale=0.3),
    "odd": dict(width=90, heads=3, kv_heads=1, dim=18, vdim=10, every=29, rheads=3, rdim=14, rvdim=9, rot=6, lheads=3, ldim=14, lvdim=9, rank=22, ff=50,
                vocab=301, logit_scale=2.0),
    "retention only": dict(width=64, types=("retention", "retention"), rheads=2, rdim=128, rvdim=[256, 320], rot=128, decay=((0.99, 0.999),), mlps=(0, 1)),
    "attention only": dict(width=64, types=("attention",), heads=2, kv_heads=2, dim=64, vdim=128, every=128, logit_scale=1.0),
    "latent only": dict(width=64, types=("latent_attention",), lheads=2, ldim=64, lvdim=64, rank=128, mlps=(0,)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_whole_prompts_portions_and_decoding(dtype, name):
    cfg = O.make_config(**CONFIGS[name])
    w = O.make_weights(cfg, 3)
    ids = tokens(333, 1)
    want = oracle(w, cfg, ids)
    core = make_core(cfg, w, dtype)
    for i, sizes in enumerate(([333], [100, 2, 2, 31, 64, 1, 1, 5, 90], [300], [2] * 40 + [253], [8, 7, 9, 15, 17, 128, 129])):
        assert close(run_portions(core, i, ids, sizes), want, dtype), sizes
        core.release(i)
    assert core.runner.graph_replays > 30


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_prompt_and_long_decoding(dtype):
    """A prompt of several query blocks and chunks, and hundreds of tokens decoded one by one with slowly fading states."""
    cfg = O.make_config(width=64, heads=4, kv_heads=2, dim=32, vdim=32, every=100, rheads=2, rdim=32, rvdim=64, rot=32, decay=((0.999, 0.9999),), lheads=2,
                        ldim=32, lvdim=32, rank=48)
    w = O.make_weights(cfg, 5)
    ids = tokens(1100, 2)
    want = oracle(w, cfg, ids)
    core = make_core(cfg, w, dtype)
    assert close(run_portions(core, 0, ids, [1100]), want, dtype)
    assert close(run_portions(core, 1, ids, [700, 3]), want, dtype)
    assert close(run_portions(core, 2, ids[:450], [3]), want[:450], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_and_reuse(dtype):
    """Unequal requests advance by unequal amounts in one batch, finished ones hand pages and state slots on."""
    from trainscale_b200.inference.trace import TraceRunner
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 4)
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
            n = min([1, 40, 2, 17, 1, 8, 80][(step + j) % 7], len(reqs[r]) - lo)
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
        assert close(torch.cat(got[r]), oracle(w, cfg, ids), dtype), r
    assert core.cache.alloc.num_free == 40 and len(core.cache.free_slots) == 3


def test_wide_decode_batch():
    """More rows than the few-row products take, odd batch sizes, captured and not."""
    from trainscale_b200.inference.batch import StepEntry
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 6)
    reqs = [tokens(5 + (7 * i) % 60, 100 + i) for i in range(45)]
    want = torch.stack([oracle(w, cfg, r)[-1] for r in reqs])
    for eager in (True, False):
        core = make_core(cfg, w, BF, seqs=45, eager=eager)
        for i, r in enumerate(reqs):
            core.execute([StepEntry(i, r[:-1], [])])
        assert close(core.execute([StepEntry(i, [r[-1]]) for i, r in enumerate(reqs)]), want, BF), eager


def test_generation_fp32_matches_oracle():
    """Greedy tokens of the engine's own entry point, with chunked prefill and preemption."""
    from trainscale_b200.inference import GenerationParams, SOTAInferenceEngine
    cfg = O.make_config(width=64)
    w = O.make_weights(cfg, 7, sharp=1.5)
    prompts = [tokens(n, n) for n in (40, 3, 77, 18)]
    want = [O.greedy(w, cfg, p, 12) for p in prompts]
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
