"""Vibepel kernels and the model on the GPU against plain fp64 PyTorch (vibepel_oracle.py and the formulas below)."""
import math

import pytest
import torch
import torch.nn.functional as F

import vibepel_oracle as O

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


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


def uniform(*shape, seed=0, lo=0.0, hi=1.0):
    return (lo + (hi - lo) * torch.rand(*shape, generator=torch.Generator().manual_seed(seed))).cuda()


def tokens(n, seed, vocab=300):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


# ---------------------------------------------------------------------------------------------- residual stream
def _rows(lens, prevs):
    """row_prev / row_next of portions of these lengths that continue state row `prevs[b]` (-1: none); portion b leaves 20 + b."""
    prev, nxt = [], []
    for b, (n, p) in enumerate(zip(lens, prevs)):
        prev += [p] + [-2] * (n - 1)
        nxt += [-1] * (n - 1) + [20 + b]
    from trainscale_b200.ops.stream import StreamRows
    return StreamRows(i32(*prev), i32(*nxt))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,lens", [(64, [5, 1, 3]), (66, [1, 1]), (100, [9]), (2048, [2, 3]), (6144, [2]), (1030, [4]), (256, [1500, 1, 1499])])
def test_postnorm_sum_and_mixes(dtype, W, lens):
    """Output norm, fp32 sum, cast or token-shift mixes: rows that start from a state row, from zero, from the row before."""
    from trainscale_b200.ops import stream
    T, n_mix, ld = sum(lens), 5, W + 7 if W % 4 else W + 8
    x, y, w = rnd(T, W, seed=1), rnd(T, W, seed=2, dtype=dtype, scale=3.0), rnd(W, seed=3, scale=0.3)
    mu, state = uniform(n_mix, W, seed=4), rnd(30, ld, seed=5)
    rows = _rows(lens, [3, -1, 7][:len(lens)])
    want = x.double() + O.norm1p(y.double(), w.double(), 1e-4)
    got, h = stream.postnorm(x, y, w, 1e-4, None, rows, None, dtype)
    assert rel(got, want) < 2e-6 and rel(h, want) < tol(dtype) and h.dtype == dtype
    before, at, prevs = state.clone(), 0, []
    got, h = stream.postnorm(x, y, w, 1e-4, mu, rows, state, dtype)
    for b, n in enumerate(lens):
        first = [3, -1, 7][b]
        head = before[first, :W].double() if first >= 0 else torch.zeros(W, dtype=torch.float64, device="cuda")
        prevs += [head[None], want[at:at + n - 1]]
        at += n
        assert torch.equal(state[20 + b, :W], got[at - 1])
    prev = torch.cat(prevs)
    assert rel(h, want[:, None] + (prev - want)[:, None] * mu.double()) < tol(dtype) and h.shape == (T, n_mix, W)
    assert torch.equal(state[:20], before[:20]) and torch.equal(state[:, W:], before[:, W:])
    sel = i32(*[T - 1, 0][:T])
    fin = stream.postnorm_final(x, y, w, mu[0], 1e-4, sel, dtype)
    assert rel(fin, O.norm1p(want, mu[0].double(), 1e-4)[sel.long()]) < tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_scaled_embedding(dtype):
    from trainscale_b200.ops import stream
    table, tok = rnd(50, 96, seed=1, dtype=dtype), torch.tensor([3, 49, 0, 3, 7], device="cuda")
    x, h = stream.scaled_embed(tok, table, 7.25, None, None, None)
    assert torch.equal(x, table[tok].float() * 7.25) and torch.equal(h, x.to(dtype))
    state, mu = rnd(30, 96, seed=2), uniform(5, 96, seed=3)
    _, h = stream.scaled_embed(tok, table, 7.25, mu, _rows([3, 2], [-1, 4]), state)
    prev = torch.cat([torch.zeros(1, 96).cuda(), x[:2], state[4:5], x[3:4]])
    assert rel(h, x[:, None] + (prev - x)[:, None] * mu) < tol(dtype)
    assert torch.equal(state[20], x[2]) and torch.equal(state[21], x[4])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(3, 40, 64), (20, 96, 128), (70, 300, 64), (600, 512, 256), (2500, 1030, 192), (5, 9, 21)])
def test_activations_of_products(dtype, M, N, K):
    from trainscale_b200.ops import gemm, grouped
    x, w = rnd(M, K, seed=1, dtype=dtype), rnd(N, K, seed=2, dtype=dtype, scale=K ** -0.5)
    z = x.double() @ w.double().t()
    for act, cap, want in ((grouped.ACT_RELU_SQUARED, 0.0, torch.relu(z).square()), (grouped.ACT_TANH, 0.0, torch.tanh(z)),
                           (grouped.ACT_SOFTCAP, 0.7, 0.7 * torch.tanh(z / 0.7))):
        assert rel(gemm.serve_linear(x, w, act=act, cap=cap), want) < tol(dtype)
        assert rel(gemm.serve_linear(x, w, torch.float32, act=act, cap=cap), want) < 4e-6
    out = torch.zeros(M, 4, N, dtype=dtype, device="cuda")
    gemm.serve_linear(x, w, out=out[:, 2])
    assert rel(out[:, 2], z) < tol(dtype) and out[:, 1].abs().sum() == 0 and out[:, 3].abs().sum() == 0


# ---------------------------------------------------------------------------------------------- windowed attention
def attention(q, k, v, scale, window, off):
    """q [Tq, H, D] at positions off .., k [Tk, G, D], v [Tk, G, V] at 0 .. in fp64."""
    rep = q.shape[1] // k.shape[1]
    s = torch.einsum("thd,jhd->htj", q, k.repeat_interleave(rep, 1)) * scale
    i, j = torch.arange(q.shape[0], device=q.device) + off, torch.arange(k.shape[0], device=q.device)
    d = i[:, None] - j[None]
    s = s.masked_fill((d < 0) | (d >= window), float("-inf"))
    return torch.einsum("htj,jhv->thv", torch.softmax(s, -1), v.repeat_interleave(rep, 1))


SHAPES = [  # H, G, dim, vdim, rot
    (5, 1, 96, 96, 40), (8, 2, 128, 128, 64), (4, 4, 64, 64, 64), (5, 5, 40, 72, 12), (24, 1, 80, 48, 16), (3, 1, 20, 12, 6),
    (4, 2, 18, 30, 18), (2, 1, 256, 128, 32), (2, 2, 200, 256, 0)]


def _shape(H, G, D, V, rot, window):
    from trainscale_b200.ops.window_attention import WindowShape
    return WindowShape(H, G, D, V, rot, window, D ** -0.5 * 1.3)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,rot", SHAPES)
def test_head_norms_rotary_and_cache_write(dtype, H, G, D, V, rot):
    from trainscale_b200.ops import window_attention as wa
    s = _shape(H, G, D, V, rot, 9)
    T, pad = 37, 8 + (-(s.q_width + s.kv_width)) % 8
    proj = rnd(T, s.q_width + s.kv_width + pad, seed=1, dtype=dtype)
    before = proj.clone()
    qn, kn = rnd(D, seed=2), rnd(D, seed=3)
    pos = torch.randint(0, 5000, (T,), generator=torch.Generator().manual_seed(4)).int().cuda()
    slots = torch.randperm(64, generator=torch.Generator().manual_seed(5))[:T].cuda()
    r = {"dims": rot, "base": 1000.0, "scaling": O.SCALING}
    f = O.frequencies(r).float().cuda()
    cache = torch.full((8, 8, s.row_width), 3.0, dtype=dtype, device="cuda")
    wa.prepare(proj, s, qn, kn, 1e-5, wa.angles(f, pos), slots, cache)

    def normed(x, w):
        return O.rotate_half(O.rms(x.double().cpu(), 1e-5) * w.double().cpu(), pos.cpu(), r)

    qw, kw = s.q_width, s.kv_heads * s.dim
    q = normed(before[:, :qw].view(T, H, D), qn).reshape(T, -1)
    k = normed(before[:, qw:qw + kw].view(T, G, D), kn).reshape(T, -1)
    loose = 6e-6 if dtype == torch.float32 else 6e-3            # fp32 angles of positions up to 5000
    assert rel(proj[:, :qw], q) < loose * 8 and rel(proj[:, qw:qw + kw], k) < loose * 8
    assert torch.equal(proj[:, qw + kw:], before[:, qw + kw:])
    rows = cache.view(-1, s.row_width)[slots]
    assert torch.equal(rows[:, :s.kv_width], proj[:, qw:qw + s.kv_width])
    assert rows[:, s.kv_width:].abs().sum() == 0
    other = torch.ones(64, dtype=torch.bool)
    other[slots.cpu()] = False
    assert (cache.view(-1, s.row_width)[other.cuda()] == 3).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,rot", SHAPES)
@pytest.mark.parametrize("bs,window,lens", [(16, 50, [1, 7, 49, 50, 51, 200]), (4, 1, [1, 5]), (64, 1000, [700, 3, 1500]), (48, 129, [128, 129, 130])])
def test_attend_rows(dtype, H, G, D, V, rot, bs, window, lens):
    """Single query rows against scattered pages; one key near the window's edge dominates, the key just outside would too."""
    from trainscale_b200.ops import window_attention as wa
    s = _shape(H, G, D, V, rot, window)
    n, nb = len(lens), max(-(-x // bs) for x in lens)
    perm = torch.randperm(n * nb + 3, generator=torch.Generator().manual_seed(1))[:n * nb].view(n, nb).int()
    cache = rnd(n * nb + 3, bs, s.row_width, seed=2, dtype=dtype)
    q = rnd(n, s.q_width + 16, seed=3, dtype=dtype)
    flat = cache.view(-1, s.row_width)
    for b, L in enumerate(lens):
        for j in (L - window, L - window - 1):                  # first visible key, last invisible one
            if j >= 0:
                slot = int(perm[b, j // bs]) * bs + j % bs
                flat[slot, :D] = q[b, :D] * 3.0
    out = torch.zeros(n, s.out_width + 8, dtype=dtype, device="cuda")
    row_seq, row_len = torch.arange(n, dtype=torch.int32, device="cuda"), i32(*lens)
    wa.attend_rows(q, s, cache, perm.cuda(), row_seq, row_len, max(lens), out, 0.75)
    for b, L in enumerate(lens):
        j = torch.arange(L)
        rows = flat[(perm[b, j // bs].long() * bs + j % bs).cuda()].double()
        k, v = rows[:, :G * D].view(L, G, D), rows[:, G * D:s.kv_width].view(L, G, V)
        want = attention(q[b:b + 1, :s.q_width].double().view(1, H, D), k, v, s.scale, window, L - 1) * 0.75
        assert rel(out[b, :s.out_width], want.reshape(-1)) < tol(dtype, 1.5), (b, L)
    assert out[:, s.out_width:].abs().sum() == 0


@pytest.mark.parametrize("H,G,D,V,rot", [x for x in SHAPES if x[2] % 8 == 0 and x[3] % 8 == 0 and x[3] <= 128])
@pytest.mark.parametrize("window,seqs", [(50, [(0, 300), (0, 1), (0, 51)]), (129, [(128, 2), (700, 260), (3, 40)]), (1, [(5, 9)]),
                                         (4000, [(0, 700), (130, 500)]), (256, [(255, 257), (256, 2), (511, 300)])])
def test_attend_portions(H, G, D, V, rot, window, seqs):
    from trainscale_b200.ops import window_attention as wa
    s = _shape(H, G, D, V, rot, window)
    assert wa.portions_supported(s)
    qs, ks, cu_q, cu_k, want = [], [], [0], [0], []
    fresh = all(start == 0 for start, _ in seqs)
    for b, (start, n) in enumerate(seqs):
        lo = max(0, start - (window - 1))
        L = start + n - lo
        q = rnd(n, s.q_width, seed=10 + b, dtype=torch.bfloat16)
        kv = rnd(L, s.row_width, seed=20 + b, dtype=torch.bfloat16)
        for i in (0, n // 2, n - 1):                            # dominant keys at both sides of the window's edge
            j = start + i - window + 1 - lo
            for jj in (j, j - 1):
                if 0 <= jj < L:
                    kv[jj, :D] = q[i, :D] * 3.0
        k, v = kv[:, :G * D].double().view(L, G, D), kv[:, G * D:s.kv_width].double().view(L, G, V)
        want.append(attention(q.double().view(n, H, D), k, v, s.scale, window, start - lo))
        qs.append(q)
        ks.append(kv)
        cu_q.append(cu_q[-1] + n)
        cu_k.append(cu_k[-1] + L)
    out = torch.zeros(cu_q[-1], s.out_width + 8, dtype=torch.bfloat16, device="cuda")
    q, rows = torch.cat(qs), torch.cat(ks)
    if fresh:
        proj = torch.cat([q, rows], 1)
        wa.attend_portions(proj, s, None, i32(*cu_q), i32(*cu_k), max(n for _, n in seqs), out, 1.25)
    else:
        wa.attend_portions(q, s, rows, i32(*cu_q), i32(*cu_k), max(n for _, n in seqs), out, 1.25)
    want = torch.cat(want).reshape(cu_q[-1], -1) * 1.25
    assert rel(out[:, :s.out_width], want) < tol(torch.bfloat16)
    worst = (out[:, :s.out_width].double() - want).abs().max() / want.abs().max()
    assert worst < 0.03 and out[:, s.out_width:].abs().sum() == 0


# ---------------------------------------------------------------------------------------------- recurrences
def _portions(lens):
    from trainscale_b200.inference.batch import Portions
    at = [0]
    for n in lens:
        at.append(at[-1] + n)
    return Portions(at, i32(*at))


PREV = [3, -1, 7, 5, -1]


def delta_case(H, G, D, V, taps, T, dtype, seed=0, strong=False):
    from trainscale_b200.ops.recurrent import DeltaShape, DeltaWeights
    s = DeltaShape(H, G, D, V, taps)
    w = DeltaWeights(rnd(s.channels, taps, seed=seed + 1, scale=0.7), rnd(H, seed=seed + 2, scale=0.5 if not strong else 3.0),
                     rnd(H, seed=seed + 3) - 3.0, rnd(V, seed=seed + 4) * 0.2 + 1)
    width = -(-s.proj_width // 8) * 8 + 8
    proj = rnd(T, width, seed=seed + 5, dtype=dtype)
    state = rnd(30, s.state_width, seed=seed + 6, scale=0.5)
    return s, w, proj, state


def delta_oracle(s, w, x, state, eps):
    """One sequence: x [T, proj_width] fp64, state row or None -> gated result [T, H V], convolution inputs, matrices."""
    C, kw, H, G = s.channels, s.kv_heads * s.dim, s.heads, s.kv_heads
    tail = torch.zeros(s.taps - 1, C, dtype=torch.float64) if state is None else state[:(s.taps - 1) * C].view(s.taps - 1, C)
    S = None if state is None else state[s.matrix_offset:s.matrix_offset + H * s.dim * s.vdim].view(H, s.dim, s.vdim)
    inp = torch.cat([tail, x[:, :C]])
    y = O.short_conv(inp, w.conv.double().cpu())[s.taps - 1:]
    grp = torch.arange(H) // (H // G)
    q = (O.unit(y[:, :kw].reshape(-1, G, s.dim)) * s.dim ** -0.5)[:, grp]
    k = O.unit(y[:, kw:2 * kw].reshape(-1, G, s.dim))[:, grp]
    at = C + s.out_width
    beta = torch.sigmoid(x[:, at:at + H])
    g = torch.exp(-torch.exp(w.A_log.double().cpu()) * F.softplus(x[:, at + H:at + 2 * H] + w.dt_bias.double().cpu()))
    o, S = O.delta_recurrence(q, k, y[:, 2 * kw:].reshape(-1, H, s.vdim), g, beta, S)
    o = O.rms(o, eps) * w.norm.double().cpu() * F.silu(x[:, C:at]).view(-1, H, s.vdim)
    return o.reshape(-1, s.out_width), inp[x.shape[0]:], S


DELTA = [(4, 2, 64, 64, 4), (4, 2, 128, 128, 4), (4, 4, 32, 24, 2), (3, 1, 96, 40, 1), (2, 1, 256, 64, 4), (2, 2, 20, 36, 6),
         (3, 3, 17, 9, 4), (2, 1, 128, 256, 2), (8, 1, 8, 8, 3), (2, 2, 256, 256, 4)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,taps", DELTA)
@pytest.mark.parametrize("lens,strong", [([5, 70, 2, 33, 8], False), ([300], False), ([41, 9], True)])
def test_delta_rule_portions(dtype, H, G, D, V, taps, lens, strong):
    """Convolution, norms, gates, scan and gated norm of portions that continue a state or start from zero, also portions
    shorter than the convolution; the states they leave.  `strong`: decays from nearly one to nearly zero."""
    from trainscale_b200.ops import recurrent
    T, ns, eps = sum(lens), 3, 1e-5
    s, w, proj, state = delta_case(H, G, D, V, taps, T + ns, dtype, strong=strong)
    rows = _rows([1] * ns + lens, [-1] * ns + PREV[:len(lens)])
    rows.next[:ns] = -1
    out = torch.zeros(T + ns, s.out_width + 8, dtype=dtype, device="cuda")
    before = state.clone()
    recurrent.delta_rule(proj[:, :s.proj_width], s, w, eps, rows, state, ns, _portions(lens), out[:, :s.out_width], 0.6)
    at = ns
    for b, n in enumerate(lens):
        x = proj[at:at + n].double().cpu()
        o, tail, S = delta_oracle(s, w, x, before[PREV[b]].double().cpu() if PREV[b] >= 0 else None, eps)
        assert rel(out[at:at + n, :s.out_width], o * 0.6) < tol(dtype, 2.0), (b, n)
        left = state[20 + ns + b]
        assert rel(left[:(taps - 1) * s.channels], tail.reshape(-1)) < 1e-6 or taps == 1
        assert rel(left[s.matrix_offset:s.matrix_offset + S.numel()], S.reshape(-1)) < 6e-6
        at += n
    assert torch.equal(state[:20], before[:20]) and out[:, s.out_width:].abs().sum() == 0


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,V,taps", DELTA)
def test_delta_rule_steps_equal_a_portion(dtype, H, G, D, V, taps):
    """Token-by-token decoding of two sequences (state rows taking turns) gives what one portion gives."""
    from trainscale_b200.ops import recurrent
    from trainscale_b200.ops.stream import StreamRows
    n, eps = 21, 1e-5
    s, w, proj, state = delta_case(H, G, D, V, taps, 2 * n, dtype, seed=40)
    outs = torch.zeros(2 * n, s.out_width, dtype=dtype, device="cuda")
    for t in range(n):
        prev = i32(-1 if t == 0 else 10 + (t & 1), 12 + (t & 1)) if t else i32(-1, 4)
        rows = StreamRows(prev, i32(10 + ((t + 1) & 1), 12 + ((t + 1) & 1)))
        x = proj[[t, n + t]][:, :s.proj_width].contiguous()
        o = torch.empty(2, s.out_width, dtype=dtype, device="cuda")
        recurrent.delta_rule(x, s, w, eps, rows, state, 2, None, o)
        outs[t], outs[n + t] = o[0], o[1]
    first = delta_case(H, G, D, V, taps, 1, dtype, seed=40)[3]
    for b, st in ((0, None), (1, first[4].double().cpu())):
        o, tail, S = delta_oracle(s, w, proj[b * n:(b + 1) * n].double().cpu(), st, eps)
        assert rel(outs[b * n:(b + 1) * n], o) < tol(dtype, 2.0)
        left = state[10 + 2 * b + (n & 1)]
        assert rel(left[s.matrix_offset:s.matrix_offset + S.numel()], S.reshape(-1)) < 6e-6


WKV = [(5, 32), (2, 64), (3, 128), (1, 256), (2, 48), (3, 20), (2, 7), (5, 8)]


def wkv_oracle(s, w, x, raw, S, eps):
    T, H, D = x.shape[0], s.heads, s.dim
    r, k, v, g = (x[:, i] for i in range(4))
    decay = torch.exp(-torch.exp(raw + w.w0.double().cpu())).view(T, H, D)
    o, S = O.wkv_recurrence(r.view(T, H, D), k.view(T, H, D), v.view(T, H, D), decay, w.u.double().cpu(), S)
    return O.rms(o, eps).reshape(T, -1) * w.norm.double().cpu() * F.silu(g), S


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D", WKV)
@pytest.mark.parametrize("lens,shift", [([5, 70, 2, 33, 8], -1.5), ([300], -5.0), ([41, 9], 3.0)])
def test_wkv_portions_and_steps(dtype, H, D, lens, shift):
    """Scan of portions and single steps; `shift` moves the decays from long memory to none at all."""
    from trainscale_b200.ops import recurrent
    from trainscale_b200.ops.recurrent import WkvShape, WkvWeights
    from trainscale_b200.ops.stream import StreamRows
    T, eps, ns = sum(lens), 1e-5, 2
    s = WkvShape(H, D, 50)
    w = WkvWeights(rnd(s.inner, seed=1) + shift, rnd(H, D, seed=2), rnd(s.inner, seed=3) * 0.2 + 1)
    x, raw = rnd(T + ns, 4, s.inner, seed=4, dtype=dtype), rnd(T + ns, s.inner, seed=5)
    state = rnd(40, s.state_width, seed=6, scale=0.5)
    before = state.clone()
    rows = _rows([1] * ns + lens, [-1, 6] + PREV[:len(lens)])
    out = torch.zeros(T + ns, s.inner, dtype=dtype, device="cuda")
    recurrent.wkv(x, raw, s, w, eps, rows, state, ns, _portions(lens), out)
    at, size = 0, H * D * D

    def matrices(row):
        return row[s.matrix_offset:s.matrix_offset + size].double().cpu().view(H, D, D)

    for b, (n, p) in enumerate(zip([1] * ns + lens, [-1, 6] + PREV)):
        o, S = wkv_oracle(s, w, x[at:at + n].double().cpu(), raw[at:at + n].double().cpu(), matrices(before[p]) if p >= 0 else None, eps)
        assert rel(out[at:at + n], o) < tol(dtype, 2.0), (b, n)
        assert rel(matrices(state[20 + b]), S) < 6e-6
        at += n
    # the first portion again, token by token
    n = min(lens[0], 25)
    outs = []
    for t in range(n):
        r = StreamRows(i32(3 if t == 0 else 30 + (t & 1)), i32(30 + ((t + 1) & 1)))
        o = torch.empty(1, s.inner, dtype=dtype, device="cuda")
        recurrent.wkv(x[ns + t:ns + t + 1], raw[ns + t:ns + t + 1], s, w, eps, r, state, 1, None, o)
        outs.append(o)
    assert rel(torch.cat(outs), out[ns:ns + n]) < tol(dtype, 2.0)


@pytest.mark.parametrize("D,H", [(64, 300), (128, 160), (64, 8)])
def test_scans_with_many_and_few_heads(D, H):
    """Grids below and above one wave take different splits of the key rows; both must give the plain scan's result."""
    from trainscale_b200.ops import recurrent
    lens = [37, 64]
    s, w, proj, state = delta_case(H, H // 2, D, D, 3, sum(lens), torch.float32, seed=60)
    rows, por = _rows(lens, [3, -1]), _portions(lens)
    qkv, gates = recurrent.delta_inputs(proj[:, :s.proj_width], s, w, rows, state, por)
    a, st = state.clone(), state.clone()
    plain = recurrent.delta_scan(qkv, gates, s, rows, a, por)
    blocked = recurrent.delta_scan(qkv, gates, s, rows, st, por, True)
    assert rel(blocked, plain) < 5e-6 and rel(st[20:22], a[20:22]) < 5e-6


# ---------------------------------------------------------------------------------------------- the model
def make_core(cfg, w, dtype, blocks=400, seqs=4, eager=False, block_size=16, budget=4096):
    from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, SchedulerConfig
    from trainscale_b200.models.vibepel import load_model
    ec = EngineConfig(model="custom", tokenizer="byte", device="cuda", dtype=str(dtype)[6:], enforce_eager=eager,
                      scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                      cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=4096))
    return EngineCore(ec, model=load_model(cfg, w, dtype, "cuda"))


def close(got, want, dtype):
    """rms over the vocabulary of the difference (mean taken off), relative to the logits' own spread.  bf16: rounding the
    operands of the products alone gives medians around 0.015 and single positions up to 0.1 in these small models."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    e = d.pow(2).mean(-1).sqrt() / want.std()
    if dtype == torch.float32:
        return e.max().item() < 3e-5
    return e.max().item() < 0.25 and (len(e) < 20 or e.median().item() < 0.03)


def run_portions(core, seq, ids, sizes):
    from trainscale_b200.inference.batch import StepEntry
    out, at, sizes = [], 0, list(sizes)
    while at < len(ids):
        n = min(sizes.pop(0) if sizes else 1, len(ids) - at)
        out.append(core.execute([StepEntry(seq, ids[at:at + n], list(range(n)))]).clone())
        at += n
    return torch.cat(out)


CONFIGS = {
    "mixed": dict(width=128, types=("wkv", "parallel", "parallel", "wkv"), heads=[6, 4, 8], kv_heads=[2, 4, 1], dim=[32, 64, 24],
                  vdim=[48, 64, 16], window=[40, 129, 17], rot=[16, 64, 10], dheads=[4, 2, 6], dkv=[2, 1, 6], ddim=[32, 64, 16],
                  dvdim=[48, 64, 8], taps=[4, 1, 2], wheads=[2, 3], wdim=[64, 32], ff=[256, 96, 200], scaling=[None, O.SCALING],
                  left_scale=[0.5, 1.0], right_scale=[1.0, 2.0], decay_rank=24),
    "odd": dict(width=90, heads=3, kv_heads=1, dim=18, vdim=10, window=33, rot=6, dheads=3, dkv=3, ddim=10, dvdim=14, taps=5, wheads=2,
                wdim=11, ff=50, decay_rank=5, vocab=301),
    "attention only": dict(width=64, types=("parallel",), heads=2, kv_heads=2, dim=64, vdim=64, window=64, rot=64, taps=4, mlp_every=2),
    "wkv only": dict(width=64, types=("wkv", "wkv"), wheads=1, wdim=64, mlp_every=2, decay_rank=8),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", CONFIGS)
def test_whole_prompts_portions_and_decoding(dtype, name):
    cfg = O.make_config(**CONFIGS[name])
    w = O.make_weights(cfg, 3)
    ids = tokens(333, 1)
    want = O.logits({k: v.double() for k, v in w.items()}, cfg, ids)
    core = make_core(cfg, w, dtype)
    for i, sizes in enumerate(([333], [100, 2, 2, 31, 64, 1, 1, 5, 90], [300], [2] * 40 + [253], [8, 7, 9, 15, 17, 128, 129])):
        assert close(run_portions(core, i, ids, sizes), want, dtype), sizes
        core.release(i)
    assert core.runner.graph_replays > 30


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_with_slow_states(dtype):
    """Few tokens at once, hundreds decoded one by one past the window, states that forget slowly."""
    cfg = O.make_config(width=64, heads=4, kv_heads=2, dim=32, vdim=32, rot=16, window=60, ddim=32, dvdim=32, wheads=2, wdim=32)
    w = O.make_weights(cfg, 5, slow=True)
    ids = tokens(420, 2)
    want = O.logits({k: v.double() for k, v in w.items()}, cfg, ids)
    core = make_core(cfg, w, dtype)
    assert close(run_portions(core, 0, ids, [3]), want, dtype)


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_and_reuse(dtype):
    """Unequal requests advance by unequal amounts in one batch, finished ones hand pages and slots on."""
    from trainscale_b200.inference.trace import TraceRunner
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 4)
    w64 = {k: v.double() for k, v in w.items()}
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
        assert close(torch.cat(got[r]), O.logits(w64, cfg, ids), dtype), r
    assert core.cache.alloc.num_free == 40 and len(core.cache.free_slots) == 3


def test_wide_decode_batch():
    """More rows than the few-row products take, odd batch sizes, captured and not."""
    from trainscale_b200.inference.batch import StepEntry
    cfg = O.make_config(**CONFIGS["mixed"])
    w = O.make_weights(cfg, 6)
    w64 = {k: v.double() for k, v in w.items()}
    reqs = [tokens(5 + (7 * i) % 60, 100 + i) for i in range(45)]
    want = [O.logits(w64, cfg, r)[-1] for r in reqs]
    for eager in (True, False):
        core = make_core(cfg, w, torch.bfloat16, seqs=45, eager=eager)
        for i, r in enumerate(reqs):
            core.execute([StepEntry(i, r[:-1], [])])
        got = core.execute([StepEntry(i, [r[-1]]) for i, r in enumerate(reqs)])
        assert close(got, torch.stack(want), torch.bfloat16)


def test_generation_fp32_matches_oracle():
    """Greedy tokens of the engine's own entry point, with chunked prefill and preemption."""
    from trainscale_b200.inference import GenerationParams, SOTAInferenceEngine
    cfg = O.make_config(width=64, types=("parallel", "wkv"), window=20)
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
    core = make_core(cfg, w, torch.bfloat16)
    ids = tokens(70, 3)
    a = core.model(torch.tensor([ids, ids[::-1]]))
    b = run_portions(core, 0, ids, [70])
    assert torch.allclose(a[0], b, atol=0.05) and math.isfinite(a.sum().item())
    _lib.raise_on_loaded_device_error()
