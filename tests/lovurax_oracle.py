"""Plain PyTorch statement of the Lovurax decoder, one function per mechanism, for the tests.

Everything is computed for one whole sequence at a time, without a cache, in the dtype of the weights it is given
(tests use float64 or float32).  Nothing here is fast and nothing is shared with the package.
"""
from __future__ import annotations

import math

import torch


# ---------------------------------------------------------------------------------------------- norms and activations
def rms(x, eps):
    """x divided by its root mean square (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm(x, w, eps):
    return rms(x, eps) * w


def silu(z):
    return z * torch.sigmoid(z)


def xielu(z, p, q):
    """z / 2 plus, right of zero, softplus(p) z^2 and, left of it, (1/2 + softplus(q)) (e^z - 1 - z)."""
    sp = lambda t: torch.log1p(torch.exp(t))                          # noqa: E731
    left = torch.expm1(torch.clamp(z, max=0.0)) - z
    return torch.where(z > 0, sp(p) * z * z, (0.5 + sp(q)) * left) + z / 2


# ---------------------------------------------------------------------------------------------- rotation, temperature, bias
def rotate_halves(x, positions, dims, base):
    """x [T, heads, d]: coordinate i turns with coordinate i + dims / 2, i < dims / 2; the others stay."""
    half = dims // 2
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=torch.float64)
    a = positions.to(torch.float64)[:, None] * f
    c, s = a.cos().to(x.dtype)[:, None], a.sin().to(x.dtype)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def temperature(n, coef, every):
    """Factor of the query at every position: grows with the logarithm of the number of whole blocks of `every` tokens."""
    return torch.tensor([1 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(n)], dtype=torch.float64)


def distance_slopes(heads):
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float64)


# ---------------------------------------------------------------------------------------------- mixers
def retention_scan(q, k, v, decay):
    """S <- decay S + k v^T, o = S^T q, one token after the other; q, k [T, H, D], v [T, H, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[2], dtype=q.dtype)
    d = torch.tensor(decay, dtype=torch.float64).to(q.dtype)[:, None, None]
    out = []
    for t in range(T):
        S = d * S + k[t, :, :, None] * v[t, :, None, :]
        out.append((S * q[t, :, :, None]).sum(1))
    return torch.stack(out)


def retention(w, p, h, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = rotate_halves((h @ w[p + "q"].t()).view(T, H, D), pos, m["rot"]["dims"], m["rot"]["base"])
    k = rotate_halves((h @ w[p + "k"].t()).view(T, H, D), pos, m["rot"]["dims"], m["rot"]["base"]) * D ** -0.5
    o = retention_scan(q, k, (h @ w[p + "v"].t()).view(T, H, V), m["decay"])
    return (rms(o, eps).reshape(T, -1) * silu(h @ w[p + "g"].t())) @ w[p + "o"].t()


def sigmoid_attend(q, k, v, scale, add):
    """Weight of a visible key: sigmoid((q . k) scale + add_h - slope_h distance); nothing is normalized."""
    T, H = q.shape[:2]
    G = k.shape[1]
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    slopes = distance_slopes(H).to(q.dtype)
    out = []
    for n in range(H):
        g = n // (H // G)
        s = (q[:, n] @ k[:, g].t()) * scale - slopes[n] * (i - j).to(q.dtype)
        out.append(torch.where(j <= i, torch.sigmoid(s + add[n]), torch.zeros_like(s)) @ v[:, g])
    return torch.stack(out, dim=1)


def attention(w, p, h, m, eps):
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = norm((h @ w[p + "q"].t()).view(T, H, D), w[p + "q.norm"], eps)
    k = norm((h @ w[p + "k"].t()).view(T, G, D), w[p + "k.norm"], eps)
    q = q * temperature(T, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None]
    o = sigmoid_attend(q, k, (h @ w[p + "v"].t()).view(T, G, V), m["scale"], w[p + "pb"])
    return (o.reshape(T, -1) * torch.sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


def latent_attention(w, p, h, m, eps):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].t()).view(T, H, D)
    c = norm(h @ w[p + "dkv"].t(), w[p + "dkv.norm"], eps)
    k, v = (c @ w[p + "uk"].t()).view(T, H, D), (c @ w[p + "uv"].t()).view(T, H, V)
    hidden = torch.arange(T)[:, None] < torch.arange(T)[None, :]
    o = torch.stack([torch.softmax((q[:, n] @ k[:, n].t() * m["scale"]).masked_fill(hidden, float("-inf")), -1) @ v[:, n]
                     for n in range(H)], dim=1)
    return (o * torch.sigmoid(h @ w[p + "g"].t())[:, :, None]).reshape(T, -1) @ w[p + "o"].t()


MIXERS = {"retention": retention, "attention": attention, "latent_attention": latent_attention}


def feed_forward(w, p, h):
    return xielu(h @ w[p + "up"].t(), *w[p + "act"]) @ w[p + "down"].t()


# ---------------------------------------------------------------------------------------------- the decoder
def residual_gate(w, p, h):
    return torch.sigmoid(h @ w[p].t() + w[p + ".b"])


def forward(w, cfg, tokens):
    """(logits [T, vocab], stream after every layer [layers, T, width]) of one sequence."""
    eps = cfg["norm"]["eps"]
    x, trail = w["embed"][torch.tensor(tokens)], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = norm(x, w[p + "norm1"], eps)
        x = x + MIXERS[layer["type"]](w, p + "mix.", h, layer["mixer"], eps) * residual_gate(w, p + "rg1", h)
        if layer["mlp"] is not None:
            h = norm(x, w[p + "norm2"], eps)
            x = x + feed_forward(w, p + "mlp.", h) * residual_gate(w, p + "rg2", h)
        trail.append(x)
    return norm(x, w["final.norm"], eps) @ w["embed"].t() * cfg["logit_scale"], torch.stack(trail)


def logits(w, cfg, tokens):
    return forward(w, cfg, tokens)[0]


def greedy(w, cfg, prompt, n):
    ids = list(prompt)
    w = {k: v.double() for k, v in w.items()}
    for _ in range(n):
        ids.append(int(logits(w, cfg, ids)[-1].argmax()))
    return ids[len(prompt):]


# ---------------------------------------------------------------------------------------------- test models
def at(v, i):
    return v[i % len(v)] if isinstance(v, (list, tuple)) else v


def make_config(types=("latent_attention", "retention", "attention", "attention"), vocab=300, width=40, heads=4, kv_heads=2, dim=10,
                vdim=12, scale=None, temp=0.4, every=7, rheads=3, rdim=12, rvdim=20, rot=8, base=200.0, decay=((0.9, 0.99, 0.6),),
                lheads=3, ldim=14, lvdim=10, rank=18, mlps=(1,), ff=56, eps=1e-5, logit_scale=0.7):
    """A configuration whose constants may be given per layer (a list is walked by layer index); `mlps` says which layers feed
    forward."""
    ls = []
    for i, kind in enumerate(types):
        s = at(scale, i) if scale is not None else None
        if kind == "retention":
            H = at(rheads, i)
            d = at(decay, i)
            mixer = {"heads": H, "dim": at(rdim, i), "vdim": at(rvdim, i), "decay": [d[h % len(d)] for h in range(H)],
                     "rot": {"base": at(base, i), "dims": at(rot, i)}}
        elif kind == "attention":
            mixer = {"heads": at(heads, i), "kv_heads": at(kv_heads, i), "dim": at(dim, i), "vdim": at(vdim, i),
                     "scale": s or at(dim, i) ** -0.5, "q_temp": {"coef": at(temp, i), "every": at(every, i)}}
        else:
            mixer = {"heads": at(lheads, i), "dim": at(ldim, i), "vdim": at(lvdim, i), "kv_rank": at(rank, i),
                     "scale": s or at(ldim, i) ** -0.5}
        ls.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": at(ff, i)} if at(mlps, i) else None})
    return {"architecture": "Lovurax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "layers": ls}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random weights (bf16-representable float32).  `sharp` scales what enters the scores, so that a wrong key changes the
    outcome instead of drowning in an even average."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def near(n, c, s=0.2):
        return c + s * torch.randn(n, generator=g)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g)}
    for i, layer in enumerate(cfg["layers"]):
        m, p, kind = layer["mixer"], f"l{i}.mix.", layer["type"]
        w[f"l{i}.norm1"] = near(W, 1.0)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        w[p + "q"] = lin(H * D, W, sharp if kind == "latent_attention" else 1.0)
        if kind == "retention":
            w[p + "k"], w[p + "v"], w[p + "g"] = lin(H * D, W), lin(H * V, W), lin(H * V, W)
        elif kind == "attention":
            G = m["kv_heads"]
            w[p + "k"], w[p + "v"], w[p + "g"] = lin(G * D, W), lin(G * V, W), lin(H * V, W)
            w[p + "q.norm"], w[p + "k.norm"], w[p + "pb"] = near(D, sharp), near(D, sharp), near(H, -2.0, 1.0)
        else:
            R = m["kv_rank"]
            w[p + "dkv"], w[p + "dkv.norm"] = lin(R, W), near(R, 1.0)
            w[p + "uk"], w[p + "uv"], w[p + "g"] = lin(H * D, R, sharp), lin(H * V, R), lin(H, W)
        w[p + "o"] = lin(W, H * V)
        w[f"l{i}.rg1"], w[f"l{i}.rg1.b"] = lin(W, W), near(W, 0.5, 0.7)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            w[f"l{i}.norm2"] = near(W, 1.0)
            w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"], w[f"l{i}.mlp.act"] = lin(ff, W), lin(W, ff), near(2, 0.3, 0.8)
            w[f"l{i}.rg2"], w[f"l{i}.rg2.b"] = lin(W, W), near(W, 0.5, 0.7)
    w["final.norm"] = near(W, 1.5)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
