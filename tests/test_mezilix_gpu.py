"""Mezilix kernels and the model on the GPU against plain fp64 PyTorch (mezilix_oracle.py and the formulas below)."""
import math

import pytest
import torch

import mezilix_oracle as O

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]


def rel(got, want):
    got, want = got.double().cpu(), want.double().cpu()
    return ((got - want).pow(2).mean().sqrt() / want.pow(2).mean().sqrt().clamp(min=1e-30)).item()


def tol(dtype, scale=1.0):
    return scale * (3e-6 if dtype == torch.float32 else 6e-3)


def rnd(*shape, seed=0, dtype=torch.float32, scale=1.0):
    g = torch.Generator().manual_seed(seed)
    return (torch.randn(*shape, generator=g) * scale).to(dtype).cuda()


def tokens(n, seed, vocab=300):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


# ---------------------------------------------------------------------------------------------- residual stream
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,T", [(64, 5), (100, 9), (66, 7), (320, 33), (1030, 4), (2048, 3), (4096, 2), (6144, 2), (256, 3000)])
def test_stream_boundary(dtype, W, T):
    """Residual sum, expert combine, depth average, norm and shift; rows that start from a state row, from zero and from the
    row before; long runs of rows per block (T = 3000)."""
    from trainscale_b200.ops import stream
    n, k, eps = 3, 2, 1e-4
    hist = rnd(n + 2, T, W, seed=1)
    x, mixer = rnd(T, W, seed=2), rnd(T, W, seed=3, dtype=dtype)
    y, wts = rnd(T * k + 5, W, seed=4, dtype=dtype), torch.rand(T, k, generator=torch.Generator().manual_seed(5)).cuda()
    dest = torch.randperm(T * k + 5, generator=torch.Generator().manual_seed(6))[:T * k].int().cuda()
    dwa, shift = rnd(n + 1, seed=7), torch.rand(W, generator=torch.Generator().manual_seed(8)).cuda()
    gain, state = torch.tensor(1.7).cuda(), rnd(7, W, seed=9)
    prev = torch.full((T,), stream.ROW_BEFORE, dtype=torch.int32)
    nxt = torch.full((T,), -1, dtype=torch.int32)
    prev[0] = stream.ROW_ZERO
    prev[T // 2], nxt[T // 2 - 1 if T > 1 else 0] = 2, 4
    nxt[T - 1] = 3
    rows = stream.StreamRows(prev.cuda(), nxt.cuda())
    state0 = state.clone()
    x2, h, hs = stream.boundary(x, mixer, (y, dest, wts), hist, dwa, n, gain, eps, shift, rows, state, dtype)
    v = x.double() + mixer.double() + (y[dest.long().view(T, k)].double() * wts.double()[..., None]).sum(1)
    avg = dwa[n].double() * v + sum(dwa[j].double() * hist[j].double() for j in range(n))
    hd = O.rms(avg, eps) * gain.double()
    before = torch.cat([torch.zeros_like(hd[:1]), hd[:-1]])
    before[T // 2] = state0[2].double()
    assert rel(hist[n], v) < 1e-6 and rel(x2, avg) < 1e-6
    assert rel(h, hd) < tol(dtype) and rel(hs, hd + (before - hd) * shift.double()) < tol(dtype)
    if T > 1:
        assert rel(state[4], hd[T // 2 - 1]) < 3e-6
    assert rel(state[3], hd[T - 1]) < 3e-6
    assert torch.equal(state[[0, 1, 2, 5, 6]], state0[[0, 1, 2, 5, 6]])
    out_rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32).cuda()
    f = stream.final(x, mixer, (y, dest, wts), hist, dwa, n, gain, eps, out_rows, dtype)
    assert rel(f, hd[out_rows.long()]) < tol(dtype)
    # no mixer output, no experts, experts in slot order
    ys = y[:T * k].contiguous()
    x3, _, _ = stream.boundary(x, None, (ys, None, wts), hist, dwa, n, gain, eps, shift, rows, state, dtype)
    v3 = x.double() + (ys.view(T, k, W).double() * wts.double()[..., None]).sum(1)
    assert rel(x3, dwa[n].double() * v3 + sum(dwa[j].double() * hist[j].double() for j in range(n))) < 1e-6
    x4, _, _ = stream.boundary(x, mixer, None, hist, dwa, n, gain, eps, shift, rows, state, dtype)
    v4 = x.double() + mixer.double()
    assert rel(x4, dwa[n].double() * v4 + sum(dwa[j].double() * hist[j].double() for j in range(n))) < 1e-6


@pytest.mark.parametrize("dtype", DTYPES)
def test_stream_embed(dtype):
    from trainscale_b200.ops import stream
    V, W, B, mp, mc = 1000, 96, 211, 2 ** 31 + 11, 40503
    table, bigram = rnd(V, W, seed=1, dtype=dtype), rnd(B + 1, W, seed=2, dtype=dtype)
    ids = tokens(11, 3, V)
    prev = [-1] + ids[:-1]
    prev[6] = 999                                   # another sequence that goes on from token 999
    row_prev = torch.tensor([-1] + [-2] * 5 + [1] + [-2] * 4, dtype=torch.int32).cuda()
    row_next = torch.tensor([-1] * 5 + [2] + [-1] * 4 + [0], dtype=torch.int32).cuda()
    hist, state = torch.zeros(2, 11, W).cuda(), rnd(3, W, seed=4)
    s1 = state[1].clone()
    shift = torch.rand(W).cuda()
    h, hs = stream.embed(torch.tensor(ids).cuda(), torch.tensor(prev, dtype=torch.int32).cuda(), table, bigram, mp, mc, hist,
                         torch.tensor(0.6).cuda(), 1e-3, shift, stream.StreamRows(row_prev, row_next), state)
    r = [B if p < 0 else (p * mp + t * mc) % B for p, t in zip(prev, ids)]
    x = table[ids].double() + bigram[r].double()
    hd = O.rms(x, 1e-3) * torch.tensor(0.6).double()
    before = torch.cat([torch.zeros_like(hd[:1]), hd[:-1]])
    before[6] = s1.double()
    assert rel(hist[0], x) < 1e-6 and rel(h, hd) < tol(dtype)
    assert rel(hs, hd + (before - hd) * shift.double()) < tol(dtype)
    assert rel(state[2], hd[5]) < 3e-6 and rel(state[0], hd[10]) < 3e-6


# ---------------------------------------------------------------------------------------------- few-row products, experts
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("M,N,K", [(1, 100, 64), (3, 48, 200), (8, 33, 1032), (13, 512, 96), (31, 17, 8), (64, 130, 2048),
                                   (70, 24, 72), (5, 20, 37)])
def test_rows_linear(dtype, M, N, K):
    from trainscale_b200.ops import grouped
    x, w = rnd(M, K, seed=1, dtype=dtype), rnd(N, K, seed=2, dtype=dtype)
    want = x.double() @ w.double().t()
    assert rel(grouped.rows_linear(x, w), want) < tol(dtype)
    assert rel(grouped.rows_linear(x, w, torch.float32), want) < 3e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,H,K,N", [(1, 3, 24, 40), (9, 2, 64, 128), (40, 5, 12, 33), (100, 2, 96, 64)])
def test_head_linear(dtype, T, H, K, N):
    from trainscale_b200.ops import grouped
    buf = rnd(T, H * (K + 8), seed=1, dtype=dtype)
    x = buf.view(T, H, K + 8)[..., :K]
    w = rnd(H, N, K, seed=2, dtype=dtype)
    want = torch.einsum("thk,hnk->thn", x.double(), w.double())
    assert rel(grouped.head_linear(x, w), want) < tol(dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,W,E,k,F", [(1, 64, 4, 2, 24), (7, 96, 12, 3, 40), (33, 64, 5, 5, 136), (64, 64, 40, 4, 64),
                                       (65, 64, 4, 2, 24), (300, 96, 12, 3, 40), (500, 128, 3, 1, 200), (90, 50, 6, 2, 17),
                                       (9, 50, 6, 2, 17), (20, 64, 1, 1, 24), (200, 64, 1, 1, 24)])
def test_routed_experts(dtype, T, W, E, k, F):
    """Router, top-k, plan and both expert products against a loop over tokens; decode-sized and prompt-sized batches."""
    from trainscale_b200.ops import gemm, grouped, moe
    x, router = rnd(T, W, seed=1, dtype=dtype), rnd(E, W, seed=2, dtype=dtype, scale=1.0 / math.sqrt(W))
    up, down = rnd(E, F, W, seed=3, dtype=dtype, scale=W ** -0.5), rnd(E, W, F, seed=4, dtype=dtype, scale=F ** -0.5)
    logits = gemm.serve_linear(x, router, torch.float32)
    z = x.double() @ router.double().t()
    assert rel(logits, z) < 3e-6
    y, dest, w = moe.routed_experts(x, logits, up, down, k, grouped.ACT_RELU_SQUARED)
    s = torch.softmax(logits.double(), -1)
    ws, idx = s.topk(k, -1)
    assert rel(w, ws) < 3e-6
    rows = dest.long().view(T, k) if dest is not None else torch.arange(T * k).view(T, k).cuda()
    got = (y[rows].double() * w.double()[..., None]).sum(1)
    want = torch.zeros_like(got)
    for j in range(k):
        h = torch.relu(torch.einsum("tw,tfw->tf", x.double(), up.double()[idx[:, j]])).square()
        want += ws[:, j, None] * torch.einsum("tf,twf->tw", h, down.double()[idx[:, j]])
    assert rel(got, want) < tol(dtype, 1.5)


def test_routed_experts_all_tokens_to_one_expert():
    from trainscale_b200.ops import grouped, moe
    for T in (50, 400):
        x, up, down = rnd(T, 64, seed=1, dtype=torch.bfloat16), rnd(6, 40, 64, seed=2, dtype=torch.bfloat16), \
            rnd(6, 64, 40, seed=3, dtype=torch.bfloat16)
        logits = torch.zeros(T, 6).cuda()
        logits[:, 4] = 9.0
        y, dest, w = moe.routed_experts(x, logits, up, down, 1, grouped.ACT_RELU_SQUARED)
        y = y if dest is None else y[dest.long()]
        want = torch.relu(x.double() @ up[4].double().t()).square() @ down[4].double().t()
        assert rel(y, want) < tol(torch.bfloat16)


# ---------------------------------------------------------------------------------------------- latent attention
def latent_setup(s, lens, bs, dtype, seed=0, sharp=3.0):
    """A paged cache of random rows in permuted pages; returns (cache, block_table, rows per sequence)."""
    g = torch.Generator().manual_seed(seed)
    nb = [-(-n // bs) for n in lens]
    perm = torch.randperm(sum(nb) + 3, generator=g)
    cache = torch.full((sum(nb) + 3, bs, s.row_width), 1e4, dtype=dtype)          # a stray key would dominate
    bt = torch.zeros(len(lens), max(nb), dtype=torch.int32)
    rows, used = [], 0
    for i, n in enumerate(lens):
        r = torch.zeros(n, s.row_width)
        r[:, :s.rank + s.rot] = torch.randn(n, s.rank + s.rot, generator=g)
        r = r.to(dtype)
        pages = perm[used:used + nb[i]]
        used += nb[i]
        bt[i, :nb[i]] = pages.int()
        for j in range(n):
            cache[pages[j // bs], j % bs] = r[j]
        rows.append(r.double())
    return cache.cuda(), bt.cuda(), rows


SHAPES = [dict(heads=2, dim=24, rot=8, vdim=16, rank=48), dict(heads=8, dim=64, rot=32, vdim=64, rank=128),
          dict(heads=20, dim=128, rot=64, vdim=128, rank=512), dict(heads=3, dim=12, rot=6, vdim=20, rank=33),
          dict(heads=17, dim=40, rot=16, vdim=24, rank=272)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [1, 16, 65, 700, 5000])
def test_attend_latent(dtype, shape, window):
    """Rows with unequal lengths around page, tile and window borders, against the softmax over exactly the visible keys."""
    from trainscale_b200.ops import latent_attention as L
    s = L.LatentShape(window=window, scale=0.2, rope_base=1e4, **shape)
    lens = [1, 16, 17, 64, 65, 66, 129, 701, 1500]
    bs = 16
    cache, bt, rows = latent_setup(s, lens, bs, dtype)
    seq_of = [8, 0, 1, 2, 3, 4, 5, 6, 7, 8]
    row_len = [900, 1, 16, 17, 64, 65, 66, 129, 701, 1500]      # sequence 8 twice: an earlier position as well
    T = len(seq_of)
    q_lat = rnd(T, s.heads, s.rank, seed=1, dtype=dtype, scale=0.5)
    proj = rnd(T, s.q_width + s.rank + s.rot, seed=2, dtype=dtype, scale=0.5)
    i32 = dict(dtype=torch.int32, device="cuda")
    got = L.attend_latent(q_lat, proj, s, cache, bt, torch.tensor(seq_of, **i32), torch.tensor(row_len, **i32), 1500)
    qr = proj[:, :s.q_width].view(T, s.heads, -1)[..., s.dim:].double().cpu()
    for t in range(T):
        n = row_len[t]
        r = rows[seq_of[t]][max(0, n - window):n]
        sc = (q_lat[t].double().cpu() @ r[:, :s.rank].t() + qr[t] @ r[:, s.rank:s.rank + s.rot].t()) * s.scale
        assert rel(got[t], torch.softmax(sc, -1) @ r[:, :s.rank]) < tol(dtype, 2.0), (t, n)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("edge", [0, 1])
def test_attend_latent_outstanding_key_at_the_window_edge(dtype, edge):
    """One key scores far above the rest: as the first visible key it decides the outcome, one before it has no effect."""
    from trainscale_b200.ops import latent_attention as L
    for window in (1, 40, 64, 65, 1000):
        s = L.LatentShape(heads=4, dim=32, rot=16, vdim=32, rank=64, window=window, scale=1.0, rope_base=1e4)
        n = 1333
        cache, bt, rows = latent_setup(s, [n], 16, dtype)
        j = n - window - edge
        if j < 0:
            continue
        q_lat = rnd(1, 4, 64, seed=3, dtype=dtype, scale=0.05)
        proj = rnd(1, s.q_width + 80, seed=4, dtype=dtype, scale=0.05)
        big = q_lat[0, 2].float() / q_lat[0, 2].float().norm() * 150.0
        cache[bt[0, j // 16], j % 16, :64] = big.to(dtype)
        r = rows[0].clone()
        r[j, :64] = big.to(dtype).double().cpu()
        i32 = dict(dtype=torch.int32, device="cuda")
        got = L.attend_latent(q_lat, proj, s, cache, bt, torch.zeros(1, **i32), torch.tensor([n], **i32), n)
        v = r[n - window:]
        qr = proj[:, :s.q_width].view(1, 4, -1)[0, :, 32:].double().cpu()
        sc = q_lat[0].double().cpu() @ v[:, :64].t() + qr @ v[:, 64:80].t()
        assert rel(got[0], torch.softmax(sc, -1) @ v[:, :64]) < tol(dtype, 2.0), window


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", SHAPES)
def test_prepare(dtype, shape):
    from trainscale_b200.ops import latent_attention as L, rope
    s = L.LatentShape(window=8, scale=0.2, rope_base=700.0, **shape)
    T, eps = 9, 1e-3
    proj = rnd(T, s.q_width + s.rank + s.rot, seed=1, dtype=dtype)
    src = proj.double().cpu()
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 5, 40000, 17], dtype=torch.int32)
    slots = torch.tensor([3, 40, 41, 8, 9, 10, 11, 12, 0])
    cache = torch.full((3, 16, s.row_width), 7.0, dtype=dtype).cuda()
    nw = rnd(s.rank, seed=2) + 1.0
    flat = L.prepare(proj, s, nw, eps, rope.rope_inv_freq(s.rot, s.rope_base).cuda(), pos.cuda(), slots.cuda(), cache, True)
    c = O.rms(src[:, s.q_width:s.q_width + s.rank], eps) * nw.double().cpu()
    kr = O.rotate_half(src[:, s.q_width + s.rank:], pos, s.rope_base)
    got = cache.view(-1, s.row_width)[slots.cuda()]
    assert torch.equal(got, flat) and bool((got[:, s.rank + s.rot:] == 0).all())
    t = 4e-3 if dtype == torch.float32 else 6e-3       # angle 40000 in 32-bit: 40000 * 2^-24
    assert rel(got[:, :s.rank], c) < tol(dtype) and rel(got[:, s.rank:s.rank + s.rot], kr) < t
    keep = [i for i in range(T) if pos[i] < 2000]
    assert rel(got[keep, s.rank:s.rank + s.rot], kr[keep]) < (6e-5 if dtype == torch.float32 else 6e-3)
    q, qs = proj[:, :s.q_width].view(T, s.heads, -1), src[:, :s.q_width].view(T, s.heads, -1)
    assert rel(q[..., :s.dim], qs[..., :s.dim]) == 0.0
    want = O.rotate_half(qs[..., s.dim:].transpose(0, 1), pos, s.rope_base).transpose(0, 1)
    assert rel(q[keep][..., s.dim:], want[keep]) < (6e-5 if dtype == torch.float32 else 6e-3)
    assert bool((cache.view(-1, s.row_width)[[1, 2, 4, 5, 47]] == 7.0).all())
    assert torch.equal(L.gather_rows(cache, slots.cuda()), got)


@pytest.mark.parametrize("shape", [dict(heads=2, dim=24, rot=8, vdim=16, rank=48), dict(heads=5, dim=64, rot=16, vdim=64, rank=64),
                                   dict(heads=2, dim=128, rot=64, vdim=128, rank=96), dict(heads=3, dim=72, rot=40, vdim=80, rank=40),
                                   dict(heads=2, dim=192, rot=64, vdim=104, rank=64)])
@pytest.mark.parametrize("window", [1, 40, 128, 129, 300, 4000])
def test_attend_expanded(shape, window):
    """Portions with and without history in one launch; queries are the last rows of their sequence's keys.  Every sequence
    gets one outstanding key per window edge, so a window that is one key off changes the result."""
    from trainscale_b200.ops import latent_attention as L
    s = L.LatentShape(window=window, scale=0.3, rope_base=1e4, **shape)
    if not L.expanded_supported(s):
        pytest.fail("shape should fit the kernel")
    seqs = [(2, 0), (2, 5), (129, 0), (200, 300), (1, 700), (300, 128), (513, 0), (77, 127)]       # (new tokens, history)
    cu_q, cu_k = [0], [0]
    for n, past in seqs:
        cu_q.append(cu_q[-1] + n)
        cu_k.append(cu_k[-1] + n + min(past, window - 1))
    Tq, Tk = cu_q[-1], cu_k[-1]
    bf = torch.bfloat16
    proj = rnd(Tq, s.q_width + s.rank + s.rot + 8 - (s.rank + s.rot) % 8, seed=1, dtype=bf)
    kv = rnd(Tk, s.heads * (s.dim + s.vdim), seed=2, dtype=bf)
    rows = rnd(Tk, s.row_width, seed=3, dtype=bf)
    for i, (n, past) in enumerate(seqs):             # aligned with the middle query of the sequence, at its first key
        a, lk = cu_k[i], cu_k[i + 1] - cu_k[i]
        qi = n // 2
        first = max(0, qi + lk - n - window + 1)
        for h in range(s.heads):
            q = proj[cu_q[i] + qi, h * (s.dim + s.rot):h * (s.dim + s.rot) + s.dim].float()
            kv[a + first, h * s.dim:(h + 1) * s.dim] = (q * 25.0 / (q.norm() * s.scale)).to(bf)
    out = torch.zeros(Tq, s.heads * s.vdim, dtype=bf).cuda()
    i32 = dict(dtype=torch.int32, device="cuda")
    L.attend_expanded(proj, kv, rows, s, torch.tensor(cu_q, **i32), torch.tensor(cu_k, **i32), 513, out)
    for i, (n, past) in enumerate(seqs):
        q = proj[cu_q[i]:cu_q[i + 1], :s.q_width].double().view(n, s.heads, -1)
        k = kv[cu_k[i]:cu_k[i + 1]].double()
        lk = k.shape[0]
        kn, v = k[:, :s.heads * s.dim].view(lk, s.heads, -1), k[:, s.heads * s.dim:].view(lk, s.heads, -1)
        kr = rows[cu_k[i]:cu_k[i + 1], s.rank:s.rank + s.rot].double()
        sc = torch.einsum("thd,shd->hts", q[..., :s.dim], kn) + torch.einsum("thd,sd->hts", q[..., s.dim:], kr)
        d = (torch.arange(n)[:, None] + lk - n - torch.arange(lk)[None]).cuda()
        sc = (sc * s.scale).masked_fill(~((d >= 0) & (d < window)), float("-inf"))
        want = torch.einsum("hts,shv->thv", torch.softmax(sc, -1), v)
        got = out[cu_q[i]:cu_q[i + 1]].view(n, s.heads, -1)
        assert rel(got, want) < 8e-3, (i, n, past)
        assert (got.double() - want).abs().max() < 6e-2, (i, n, past)


# ---------------------------------------------------------------------------------------------- the model
def engine(cfg, w, dtype="float32", blocks=256, seqs=4, eager=False, budget=512, block_size=16):
    from trainscale_b200.inference import CacheConfig, EngineConfig, EngineCore, SchedulerConfig
    from trainscale_b200.models.mezilix import load_model
    dt = getattr(torch, dtype)
    return EngineCore(EngineConfig(model="custom", tokenizer="byte", device="cuda", dtype=dtype, enforce_eager=eager,
                                   scheduler=SchedulerConfig(max_num_seqs=seqs, max_num_batched_tokens=budget),
                                   cache=CacheConfig(block_size=block_size, num_gpu_blocks=blocks, max_model_len=2048)),
                      model=load_model(cfg, w, dt, "cuda"))


CASES = {
    "unlike": dict(layers=3, heads=[2, 3, 1], dim=[24, 12, 40], rot_dim=[8, 4, 16], vdim=[16, 20, 8], kv_rank=[40, 24, 33],
                   window=[7, 19, 50], experts=[5, 3, 4], top=[2, 1, 4], ff=[24, 10, 17], base=[500.0, 10000.0, 50.0]),
    "tiles": dict(width=192, layers=2, heads=[4, 18], dim=[64, 48], rot_dim=[32, 16], vdim=[64, 32], kv_rank=[128, 80],
                  window=[33, 129], experts=[8, 70], top=[3, 6], ff=[104, 64]),
    "odd": dict(width=50, layers=2, kv_rank=7, dim=3, rot_dim=2, vdim=5, ff=9, mlp_every=2),
}


def portions(core, seq, ids, sizes):
    from trainscale_b200.inference.batch import StepEntry
    out, at, sizes = [], 0, list(sizes)
    while at < len(ids):
        n = min(sizes.pop(0) if sizes else 1, len(ids) - at)
        out.append(core.execute([StepEntry(seq, ids[at:at + n], list(range(n)))]).clone())
        at += n
    core.release(seq)
    return torch.cat(out)


def model_tol(dtype):
    # bf16: single logits rows move by a few percent when the roundings of a layer differ; fp32 is the sharp test
    return 2e-5 if dtype == "float32" else 4e-2


def oracle64(w, cfg, ids):
    return O.logits({k: v.double() for k, v in w.items()}, cfg, ids)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("case", CASES)
def test_prompt_portions_and_decoding(case, dtype):
    """Whole prompt, portions down to two tokens, and token-by-token decoding (captured graphs) against the oracle."""
    cfg = O.make_config(**CASES[case])
    w = O.make_weights(cfg, 1, 1.5)
    core = engine(cfg, w, dtype)
    ids = tokens(190, 2)
    want = oracle64(w, cfg, ids)
    for k, sizes in enumerate(([190], [100, 2, 3, 2, 40, 30, 13], [2] * 95, [150], [64, 16, 48, 62])):
        assert rel(portions(core, k, ids, sizes), want) < model_tol(dtype), sizes
    assert core.runner.graph_replays > 30
    from trainscale_b200.ops import _lib
    _lib.raise_on_loaded_device_error()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_mixed_batches_reuse_pages_and_slots(dtype):
    """Portions of some requests beside single tokens of others, in a pool that holds only a few requests at a time."""
    from trainscale_b200.inference.trace import TraceRunner
    cfg = O.make_config(**CASES["tiles"])
    w = O.make_weights(cfg, 3, 1.5)
    core = engine(cfg, w, dtype, blocks=40, seqs=3)
    reqs = {f"r{i}": tokens(n, 10 + i) for i, n in enumerate([137, 5, 222, 1, 148, 13, 90, 2])}
    waiting, live, at, got, step = list(reqs), [], {}, {r: [] for r in reqs}, 0
    runner = TraceRunner(core)
    while waiting or live:
        while waiting and len(live) < 3:
            live.append(waiting.pop(0))
        entries, end = [], []
        for j, r in enumerate(live):
            lo = at.get(r, 0)
            n = min([1, 29, 2, 64, 1, 1, 3, 16][(step + 3 * j) % 8], len(reqs[r]) - lo)
            if (step + j) % 7 == 4:
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
    assert core.cache.alloc.num_free == 40 and len(core.cache.free_slots) == 3
    for r, ids in reqs.items():
        assert rel(torch.cat(got[r]), oracle64(w, cfg, ids)) < model_tol(dtype), r


def test_batch_rows_equal_single_rows():
    """A request's logits alone and inside a batch of others differ by rounding only (fp32)."""
    from trainscale_b200.inference.batch import StepEntry
    cfg = O.make_config(**CASES["tiles"])
    w = O.make_weights(cfg, 4, 1.5)
    core = engine(cfg, w, "float32", seqs=8)
    lens = [1, 80, 2, 33, 1, 150]
    ids = [tokens(n, 40 + n + i) for i, n in enumerate(lens)]
    got = core.execute([StepEntry(i, t, None) for i, t in enumerate(ids)])
    for i, t in enumerate(ids):
        alone = core.execute([StepEntry(100, t, None)])
        core.release(100)
        assert rel(got[i:i + 1], alone) < 1e-5


def test_long_decoding_matches_oracle():
    cfg = O.make_config(**CASES["tiles"], base=300.0)
    w = O.make_weights(cfg, 5, 1.5)
    core = engine(cfg, w, "float32")
    ids = tokens(400, 6)
    assert rel(portions(core, 0, ids, [3]), oracle64(w, cfg, ids)) < 2e-5


def test_greedy_generation_matches_oracle():
    """Through the engine's own scheduler: ample cache, small token budget, and a pool that forces preemption."""
    from trainscale_b200.inference import GenerationParams
    cfg = O.make_config(**CASES["tiles"])
    w = O.make_weights(cfg, 7, 1.5)
    prompts = [tokens(n, 60 + n) for n in (70, 3, 41, 18)]
    want = [O.greedy({k: v.double() for k, v in w.items()}, cfg, p, 10) for p in prompts]
    for kw in (dict(), dict(eager=True), dict(budget=11), dict(blocks=9)):
        core = engine(cfg, w, "float32", **kw)
        rs = [core.add_request(p, GenerationParams(max_tokens=10, temperature=0.0, ignore_eos=True)) for p in prompts]
        while core.has_unfinished():
            core.step()
        assert [r.output_ids for r in rs] == want, kw
        if not kw:
            assert core.runner.graph_replays >= 8


def test_bf16_rejects_nothing_it_should_run():
    """Which kernels take which shapes: tensor-core paths for multiples of eight, the general kernels for the rest."""
    from trainscale_b200.ops import latent_attention as L
    ok = L.LatentShape(4, 64, 16, 64, 128, 40, 0.1, 1e4)
    assert L.expanded_supported(ok)
    assert not L.expanded_supported(L.LatentShape(4, 12, 4, 20, 24, 40, 0.1, 1e4))
    assert not L.expanded_supported(L.LatentShape(4, 64, 16, 256, 128, 40, 0.1, 1e4))


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_wide_decode_batch(dtype):
    """More sequences than the few-row kernels take: tensor-core products, grouped experts and a padded captured batch."""
    from trainscale_b200.inference.batch import StepEntry
    cfg = O.make_config(**CASES["tiles"])
    w = O.make_weights(cfg, 8, 1.5)
    core = engine(cfg, w, dtype, seqs=45, blocks=45 * 8)
    ids = [tokens(20 + 2 * i, 200 + i) for i in range(45)]
    for a in range(0, 45, 15):
        core.execute([StepEntry(i, ids[i][:-3], []) for i in range(a, a + 15)])
    for k in (3, 2, 1):
        got = core.execute([StepEntry(i, [t[-k]], None) for i, t in enumerate(ids)]).clone()
    assert core.runner.graph_replays == 3
    for i in range(0, 45, 6):
        assert rel(got[i], oracle64(w, cfg, ids[i])[-1]) < model_tol(dtype), i


def test_trace_program(tmp_path):
    """bin/trace_run as a process of its own: a directory with config.json and weights, steps on stdin, logits in files."""
    import json
    import subprocess
    from pathlib import Path

    import numpy as np
    from trainscale_b200.hub import ModelSerializer
    cfg = O.make_config(**CASES["unlike"])
    w = O.make_weights(cfg, 9, 1.5)
    (tmp_path / "model").mkdir()
    (tmp_path / "model" / "config.json").write_text(json.dumps(cfg))
    ModelSerializer().save({k: v.to(torch.bfloat16) for k, v in w.items()}, tmp_path / "model")
    a, b = tokens(40, 1), tokens(9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b, "want": [8, 0]}, {"id": "a", "tokens": a[30:31], "want": [0]}],
              "end": ["b"]},
             {"step": 2, "entries": [{"id": "a", "tokens": a[31:], "want": [2, 8]}], "end": ["a"]}]
    for dtype in ("float32", "bfloat16"):
        out = tmp_path / dtype
        out.mkdir()
        r = subprocess.run([str(Path(__file__).resolve().parent.parent / "bin" / "trace_run"), "--model", str(tmp_path / "model"),
                            "--dtype", dtype, "--out", str(out), "--max-tokens", "128"],
                           input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=240)
        assert r.returncode == 0, r.stderr[-2000:]
        assert r.stdout.split("\n")[:3] == ["done 0", "done 1", "done 2"] and not (out / "0.f32").exists()
        la, lb = oracle64(w, cfg, a), oracle64(w, cfg, b)
        for step, want in ((1, torch.stack([lb[8], lb[0], la[30]])), (2, torch.stack([la[33], la[39]]))):
            got = torch.from_numpy(np.fromfile(out / f"{step}.f32", dtype="<f4").copy()).view(want.shape)
            assert rel(got, want) < model_tol(dtype)
