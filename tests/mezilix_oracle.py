"""Plain PyTorch statement of the Mezilix decoder, one function per mechanism, for the tests.

Everything is computed for one whole sequence at a time, without a cache, in the dtype of the weights it is given
(tests use float64 or float32).  Nothing here is fast and nothing is shared with the package.
"""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    """x divided by its root mean square (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def scalar_norm(x, gain, eps):
    return rms(x, eps) * gain


def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """Row of the pair table for every position; the sequence's first token takes the extra last row."""
    rows = [buckets]
    for prev, cur in zip(tokens[:-1], tokens[1:]):
        rows.append((prev * mul_prev + cur * mul_cur) % buckets)
    return rows


def embed(w, tokens, cfg):
    bg = cfg["embedding"]["bigram"]
    rows = bigram_rows(tokens, bg["buckets"], bg["mul_prev"], bg["mul_cur"])
    return w["embed"][torch.tensor(tokens)] + w["bigram"][torch.tensor(rows)]


def token_shift(h, mu):
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def rotate_half(x, positions, base):
    """x [..., T, d]: coordinate i turns with coordinate i + d/2 by the angle position * base^(-2i/d)."""
    d = x.shape[-1]
    half = d // 2
    freq = torch.tensor([base ** (-2.0 * i / d) for i in range(half)], dtype=torch.float64)
    ang = positions.to(torch.float64)[:, None] * freq
    c, s = ang.cos().to(x.dtype), ang.sin().to(x.dtype)
    u, v = x[..., :half], x[..., half:]
    return torch.cat([u * c - v * s, v * c + u * s], dim=-1)


def window_mask(n, size):
    i = torch.arange(n)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size)


def latent_attention(w, p, h, m, eps):
    T = h.shape[0]
    H, dim, rot, vdim, rank = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].t()).view(T, H, dim + rot)
    down = h @ w[p + "dkv"].t()
    c = rms(down[:, :rank], eps) * w[p + "dkv.norm"]
    k_rot = rotate_half(down[:, rank:], pos, m["rot"]["base"])
    q_rot = rotate_half(q[..., dim:].transpose(0, 1), pos, m["rot"]["base"])            # [H, T, rot]
    k = (c @ w[p + "uk"].t()).view(T, H, dim)
    v = (c @ w[p + "uv"].t()).view(T, H, vdim)
    s = torch.einsum("thd,shd->hts", q[..., :dim], k) + torch.einsum("htd,sd->hts", q_rot, k_rot)
    s = (s * m["scale"]).masked_fill(~window_mask(T, m["mask"]["size"]), float("-inf"))
    o = torch.einsum("hts,shv->thv", torch.softmax(s, dim=-1), v)
    return o.reshape(T, H * vdim) @ w[p + "o"].t()


def expert(w, p, h):
    return torch.relu(h @ w[p + "up"].t()).square() @ w[p + "down"].t()


def mixture(w, p, h, mlp):
    E, top = mlp["router"]["experts"], mlp["router"]["top"]
    s = torch.softmax(h @ w[p + "router"].t(), dim=-1)
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        order = sorted(range(E), key=lambda e: -float(s[t, e]))[:top]
        for e in order:
            out[t] += s[t, e] * expert(w, f"{p}e{e}.", h[t])
    return out


def depth_average(coeff, history):
    return sum(a * x for a, x in zip(coeff, history))


def layers(w, cfg, tokens):
    """Residual stream after every layer [L, T, width]."""
    eps = cfg["norm"]["eps"]
    history = [embed(w, tokens, cfg)]
    x, out = history[0], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = scalar_norm(x, w[p + "norm1"], eps)
        y = latent_attention(w, p + "mix.", token_shift(h, w[p + "shift"]), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            y = y + mixture(w, p + "mlp.", h, layer["mlp"])
        history.append(x + y)
        x = depth_average(w[p + "dwa"], history)
        out.append(x)
    return torch.stack(out) if out else history[0].unsqueeze(0)


def logits(w, cfg, tokens):
    """Logits of every position [T, vocab]."""
    x = layers(w, cfg, tokens)[-1]
    return scalar_norm(x, w["final.norm"], cfg["norm"]["eps"]) @ w["head"].t()


def greedy(w, cfg, tokens, n):
    ids = list(tokens)
    for _ in range(n):
        ids.append(int(logits(w, cfg, ids)[-1].argmax()))
    return ids[len(tokens):]


# ---------------------------------------------------------------------------------------------- test models
def make_config(width=64, vocab=300, heads=2, dim=24, rot_dim=8, vdim=16, kv_rank=40, window=7, experts=5, top=2, ff=24,
                layers=2, buckets=53, mul_prev=13, mul_cur=5, base=500.0, scale=None, eps=1e-5, mlp_every=1):
    """A configuration dictionary as a checkpoint's config.json holds it.  `heads`, `dim`, `window` ... may be lists
    (one value per layer); `mlp_every` > 1 leaves layers without a feed-forward in between."""
    def at(v, i):
        return v[i % len(v)] if isinstance(v, (list, tuple)) else v

    ls = []
    for i in range(layers):
        d, r = at(dim, i), at(rot_dim, i)
        ls.append({"type": "latent_attention",
                   "mixer": {"heads": at(heads, i), "dim": d, "rot_dim": r, "vdim": at(vdim, i), "kv_rank": at(kv_rank, i),
                             "mask": {"size": at(window, i)}, "rot": {"base": at(base, i), "dims": r},
                             "scale": at(scale, i) if scale is not None else (d + r) ** -0.5},
                   "mlp": None if i % mlp_every else
                   {"kind": "moe", "expert": {"ff": at(ff, i)}, "router": {"experts": at(experts, i), "top": at(top, i)}}})
    return {"architecture": "Mezilix", "vocab": vocab, "width": width, "norm": {"eps": eps},
            "embedding": {"bigram": {"buckets": buckets, "mul_prev": mul_prev, "mul_cur": mul_cur}}, "layers": ls}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random weights (bf16-representable float32).  `sharp` scales the query projections, so that a wrong key changes
    the outcome instead of drowning in an even average."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g),
         "bigram": torch.randn(cfg["embedding"]["bigram"]["buckets"] + 1, W, generator=g) * 0.7}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}."
        w[p + "norm1"] = torch.tensor(1.0 + 0.2 * torch.randn((), generator=g).item())
        w[p + "shift"] = torch.rand(W, generator=g)
        w[p + "dwa"] = torch.cat([0.3 * torch.randn(i + 1, generator=g), torch.ones(1)])
        w[p + "mix.q"] = lin(m["heads"] * (m["dim"] + m["rot_dim"]), W, sharp)
        w[p + "mix.dkv"] = lin(m["kv_rank"] + m["rot_dim"], W)
        w[p + "mix.dkv.norm"] = 1.0 + 0.2 * torch.randn(m["kv_rank"], generator=g)
        w[p + "mix.uk"] = lin(m["heads"] * m["dim"], m["kv_rank"])
        w[p + "mix.uv"] = lin(m["heads"] * m["vdim"], m["kv_rank"])
        w[p + "mix.o"] = lin(W, m["heads"] * m["vdim"])
        if layer["mlp"] is not None:
            E, ff = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            w[p + "mlp.router"] = lin(E, W, 2.0)
            for e in range(E):
                w[f"{p}mlp.e{e}.up"], w[f"{p}mlp.e{e}.down"] = lin(ff, W), lin(W, ff, 1.5)
    w["final.norm"] = torch.tensor(1.3)
    w["head"] = lin(cfg["vocab"], W, 2.0)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
