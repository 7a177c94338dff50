"""Plain PyTorch statement of the Kabulix decoder, one function per mechanism, for the tests.

Everything is computed for one whole sequence at a time, without a cache, in the dtype of the weights it is given
(tests use float64 or float32).  Nothing here is fast and nothing is shared with the package.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


# ---------------------------------------------------------------------------------------------- norms
def rms(x, eps):
    """x divided by its root mean square (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm1p(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


# ---------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """Angle per position of every rotated pair; with `scaling`, long wavelengths are stretched by its factor (YaRN)."""
    n, base, s = rot["dims"], rot["base"], rot.get("scaling")
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if s:
        def index(turns):                 # pair index whose wavelength makes `turns` turns over the original length
            return n * math.log(s["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
        lo, hi = max(math.floor(index(s["fast"])), 0), min(math.ceil(index(s["slow"])), n - 1)
        for i in range(n // 2):
            t = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
            f[i] = f[i] / s["factor"] * t + f[i] * (1 - t)
    return torch.tensor(f, dtype=torch.float64)


def magnitude(rot):
    """Factor of both cosine and sine."""
    return 0.1 * math.log(rot["scaling"]["factor"]) + 1 if rot.get("scaling") else 1.0


def rotate_pairs(x, positions, rot):
    """x [T, heads, d]: of the first `dims` coordinates, each even one turns with the odd one behind it."""
    n = rot["dims"]
    a = positions.to(torch.float64)[:, None] * frequencies(rot)
    c = (a.cos() * magnitude(rot)).to(x.dtype)[:, None]
    s = (a.sin() * magnitude(rot)).to(x.dtype)[:, None]
    u, v = x[..., 0:n:2], x[..., 1:n:2]
    turned = torch.stack([u * c - v * s, v * c + u * s], dim=-1).flatten(-2)
    return torch.cat([turned, x[..., n:]], dim=-1)


# ---------------------------------------------------------------------------------------------- masks
def window_mask(n, size, keep=0):
    """[query, key]: the last `size` positions, and the first `keep` of the sequence."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep))


def chunk_mask(n, size):
    """[query, key]: earlier positions of the same chunk of `size`."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def attend(q, k, v, scale, visible):
    """q [Tq, H, D], k [Tk, G, D], v [Tk, G, V], visible [Tq, Tk] -> [Tq, H, V]; consecutive heads share a key head."""
    H, G = q.shape[1], k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = ((q[:, h] @ k[:, g].t()) * scale).masked_fill(~visible, float("-inf"))
        out.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.stack(out, dim=1)


# ---------------------------------------------------------------------------------------------- mixers
def sink_attention(w, p, h, m, eps):
    """Biased projections, values = projected keys, head norms, rotary pairs, window with kept first tokens."""
    T, H, G, D = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w[p + "q"].t() + w[p + "q.b"]).view(T, H, D)
    k = (h @ w[p + "k"].t() + w[p + "k.b"]).view(T, G, D)
    pos = torch.arange(T)
    qr = rotate_pairs(rms(q, eps) * w[p + "q.norm"], pos, m["rot"])
    kr = rotate_pairs(rms(k, eps) * w[p + "k.norm"], pos, m["rot"])
    o = attend(qr, kr, k, m["scale"], window_mask(T, m["mask"]["size"], m["mask"]["keep_first"]))
    return o.reshape(T, -1) @ w[p + "o"].t()


def latent_attention(w, p, h, m, eps):
    """Keys and values expanded from a normed latent, one rotated key part for all heads, gate per value element."""
    T, H, D, R, V, K = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].t()).view(T, H, D + R)
    qn, qr = q[..., :D], rotate_pairs(q[..., D:], pos, m["rot"])
    down = h @ w[p + "dkv"].t()
    c = rms(down[:, :K], eps) * w[p + "dkv.norm"]
    kr = rotate_pairs(down[:, None, K:], pos, m["rot"])
    kn = (c @ w[p + "uk"].t()).view(T, H, D)
    v = (c @ w[p + "uv"].t()).view(T, H, V)
    o = attend(torch.cat([qn, qr], -1), torch.cat([kn, kr.expand(T, H, R)], -1), v, m["scale"], window_mask(T, m["mask"]["size"]))
    return (o.reshape(T, -1) * torch.sigmoid(h @ w[p + "g"].t())) @ w[p + "o"].t()


def chunk_attention(w, p, h, m, eps):
    """No positions, no norms; a chunk sees only itself; gate per head."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w[p + "q"].t()).view(T, H, D)
    k = (h @ w[p + "k"].t()).view(T, G, D)
    v = (h @ w[p + "v"].t()).view(T, G, V)
    o = attend(q, k, v, m["scale"], chunk_mask(T, m["mask"]["size"]))
    return (o * torch.sigmoid(h @ w[p + "g"].t())[..., None]).reshape(T, -1) @ w[p + "o"].t()


MIXERS = {"attention": sink_attention, "latent_attention": latent_attention, "attention_2": chunk_attention}


# ---------------------------------------------------------------------------------------------- feed-forwards
def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def gated(w, p, h, act):
    return (act(h @ w[p + "gate"].t()) * (h @ w[p + "up"].t())) @ w[p + "down"].t()


def group_routing(z, top, count, keep):
    """Router logits [T, E] -> chosen experts [T, top] and their weights: the best `keep` of `count` groups of neighbours by
    the sum of a group's two largest sigmoids, then the best `top` experts of those groups."""
    s = torch.sigmoid(z)
    T, E = s.shape
    groups = s.view(T, count, E // count)
    value = groups.topk(min(2, E // count), dim=-1).values.sum(-1)
    ids, weights = [], []
    for t in range(T):
        best = value[t].topk(keep).indices.tolist()
        allowed = [e for e in range(E) if e // (E // count) in best]
        pick = sorted(allowed, key=lambda e: -float(s[t, e]))[:top]
        ids.append(pick)
        weights.append(s[t, pick] / (s[t, pick].sum() + 1e-20))
    return torch.tensor(ids), torch.stack(weights)


def experts(w, p, h, f):
    r = f["router"]
    ids, weights = group_routing(h @ w[p + "router"].t(), r["top"], r["groups"]["count"], r["groups"]["keep"])
    rows = []
    for t in range(h.shape[0]):
        rows.append(sum(weights[t, j] * gated(w, f"{p}e{int(e)}.", h[t], F.silu) for j, e in enumerate(ids[t])))
    return torch.stack(rows) + torch.sigmoid(h @ w[p + "shared.sg"].t()) * gated(w, p + "shared.", h, F.silu)


def feed_forward(w, p, h, f):
    return gated(w, p, h, gelu_tanh) if f["kind"] == "dense" else experts(w, p, h, f)


# ---------------------------------------------------------------------------------------------- the decoder
def layers(w, cfg, tokens):
    """Residual stream after every layer [L, T, width]."""
    eps = cfg["norm"]["eps"]
    x, out = w["embed"][torch.tensor(tokens)], []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](w, p + "mix.", norm1p(x, w[p + "norm1"], eps), layer["mixer"], eps)
        if layer.get("mlp") is not None:
            x = x + feed_forward(w, p + "mlp.", norm1p(x, w[p + "norm2"], eps), layer["mlp"])
        out.append(x)
    return torch.stack(out)


def logits(w, cfg, tokens):
    """Logits of every position [T, vocab]."""
    return norm1p(layers(w, cfg, tokens)[-1], w["final.norm"], cfg["norm"]["eps"]) @ w["embed"].t()


def greedy(w, cfg, tokens, n):
    ids = list(tokens)
    for _ in range(n):
        ids.append(int(logits(w, cfg, ids)[-1].argmax()))
    return ids[len(tokens):]


# ---------------------------------------------------------------------------------------------- test models
def at(v, i):
    """Value of layer i: lists hold one value per layer (repeated)."""
    return v[i % len(v)] if isinstance(v, (list, tuple)) else v


SCALING = {"factor": 3.0, "original": 60, "fast": 8.0, "slow": 1.0}


def make_config(width=48, vocab=300, types=("attention", "attention_2", "latent_attention"), heads=4, kv_heads=2, dim=16, vdim=24,
                window=9, keep=3, chunk=11, rot=8, base=500.0, scaling=SCALING, scale=None, lheads=3, ldim=12, lrot=8, lvdim=10,
                rank=20, lwindow=13, mlps=("dense", "moe"), ff=40, experts=6, top=2, groups=3, keep_groups=2, expert_ff=20,
                shared_ff=28, eps=1e-5):
    """A configuration dictionary as a checkpoint's config.json holds it.  Sizes may be lists (one value per layer); `mlps`
    names a feed-forward per layer: dense, moe or None."""
    ls = []
    for i, kind in enumerate(types):
        s = at(scale, i) if scale is not None else None
        if kind == "latent_attention":
            r = {"base": at(base, i), "dims": at(lrot, i)}
            if at(scaling, i):
                r["scaling"] = dict(at(scaling, i))
            mixer = {"heads": at(lheads, i), "dim": at(ldim, i), "rot_dim": at(lrot, i), "vdim": at(lvdim, i), "kv_rank": at(rank, i),
                     "mask": {"size": at(lwindow, i)}, "rot": r, "scale": s or (at(ldim, i) + at(lrot, i)) ** -0.5}
        else:
            mixer = {"heads": at(heads, i), "kv_heads": at(kv_heads, i), "dim": at(dim, i), "scale": s or at(dim, i) ** -0.5}
            if kind == "attention":
                mixer |= {"vdim": at(dim, i), "mask": {"size": at(window, i), "keep_first": at(keep, i)},
                          "rot": {"base": at(base, i), "dims": at(rot, i)}}
            else:
                mixer |= {"vdim": at(vdim, i), "mask": {"size": at(chunk, i)}}
        f = at(mlps, i)
        mlp = None
        if f == "dense":
            mlp = {"kind": "dense", "ff": at(ff, i)}
        elif f == "moe":
            mlp = {"kind": "moe", "expert": {"ff": at(expert_ff, i)}, "shared": {"ff": at(shared_ff, i)},
                   "router": {"experts": at(experts, i), "top": at(top, i), "groups": {"count": at(groups, i), "keep": at(keep_groups, i)}}}
        ls.append({"type": kind, "mixer": mixer, "mlp": mlp})
    return {"architecture": "Kabulix", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": ls}


def make_weights(cfg, seed=0, sharp=1.0):
    """Random weights (bf16-representable float32).  `sharp` scales what enters the scores, so that a wrong key changes the
    outcome instead of drowning in an even average."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def near(n, c, s=0.2):
        return c + s * torch.randn(n, generator=g)

    def product(p, ff):
        w[p + "gate"], w[p + "up"], w[p + "down"] = lin(ff, W), lin(ff, W), lin(W, ff)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g)}
    for i, layer in enumerate(cfg["layers"]):
        m, p, kind = layer["mixer"], f"l{i}.mix.", layer["type"]
        w[f"l{i}.norm1"] = near(W, 0.0)
        H, D, V = m["heads"], m["dim"], m["vdim"]
        if kind == "latent_attention":
            R, K = m["rot_dim"], m["kv_rank"]
            w[p + "q"], w[p + "dkv"], w[p + "g"] = lin(H * (D + R), W, sharp), lin(K + R, W), lin(H * V, W)
            w[p + "dkv.norm"], w[p + "uk"], w[p + "uv"] = near(K, 1.0), lin(H * D, K, sharp), lin(H * V, K)
        else:
            G = m["kv_heads"]
            w[p + "q"], w[p + "k"] = lin(H * D, W, sharp), lin(G * D, W)
            if kind == "attention":
                w[p + "q.b"], w[p + "k.b"] = near(H * D, 0.0), near(G * D, 0.0)
                w[p + "q.norm"], w[p + "k.norm"] = near(D, sharp), near(D, sharp)
            else:
                w[p + "v"], w[p + "g"] = lin(G * V, W), lin(H, W)
        w[p + "o"] = lin(W, H * V)
        f = layer["mlp"]
        if f is not None:
            w[f"l{i}.norm2"] = near(W, 0.0)
            q = f"l{i}.mlp."
            if f["kind"] == "dense":
                product(q, f["ff"])
            else:
                for e in range(f["router"]["experts"]):
                    product(f"{q}e{e}.", f["expert"]["ff"])
                w[q + "router"] = lin(f["router"]["experts"], W, 2.0)
                product(q + "shared.", f["shared"]["ff"])
                w[q + "shared.sg"] = lin(1, W)
    w["final.norm"] = near(W, 0.5)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}


def close_calls(w, cfg, tokens, margin):
    """Positions where a router's last chosen and first rejected expert (or group) differ by less than `margin`, so that
    rounding may turn the choice."""
    eps, bad = cfg["norm"]["eps"], set()
    x = w["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        p, f = f"l{i}.", layer["mlp"]
        x = x + MIXERS[layer["type"]](w, p + "mix.", norm1p(x, w[p + "norm1"], eps), layer["mixer"], eps)
        if f is None:
            continue
        h = norm1p(x, w[p + "norm2"], eps)
        if f["kind"] == "moe":
            r = f["router"]
            s = torch.sigmoid(h @ w[p + "mlp.router"].t())
            size = r["experts"] // r["groups"]["count"]
            value = s.unflatten(1, (-1, size)).topk(min(2, size), -1).values.sum(-1).sort(-1, descending=True)
            k = r["groups"]["keep"]
            gap = torch.full((len(tokens),), 1.0, dtype=s.dtype)
            if k < r["groups"]["count"]:
                gap = value.values[:, k - 1] - value.values[:, k]
            kept = torch.zeros_like(value.values, dtype=torch.bool).scatter_(1, value.indices[:, :k], True)
            left = s.masked_fill(~kept.repeat_interleave(size, 1), -1.0).sort(-1, descending=True).values
            if r["top"] < k * size:
                gap = torch.minimum(gap, left[:, r["top"] - 1] - left[:, r["top"]])
            bad |= set((gap < margin).nonzero().flatten().tolist())
        x = x + feed_forward(w, p + "mlp.", h, f)
    return sorted(bad)
