"""Plain PyTorch statement of the Vibepel decoder, one function per mechanism, for the tests.

Everything is computed for one whole sequence at a time, without a cache, in the dtype of the weights it is given
(tests use float64 or float32).  Recurrences run token by token.  Nothing here is fast and nothing is shared with the
package.
"""
from __future__ import annotations

import math

import torch
import torch.nn.functional as F


def rms(x, eps):
    """x divided by its root mean square (eps inside the root)."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm1p(x, w, eps):
    """RMS norm whose weight is stored around zero."""
    return rms(x, eps) * (1 + w)


def embed(w, tokens, cfg):
    return w["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]


# ---------------------------------------------------------------------------------------------- WKV time mixing
def token_mix(h, mu):
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (prev - h) * mu


def wkv_recurrence(r, k, v, decay, u, state=None):
    """r, k, decay [T, H, D], v [T, H, V], u [H, D] -> o [T, H, V] and the last state [H, D, V]."""
    T, H, D = r.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=r.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S + u[:, :, None] * kv, r[t]))
        S = decay[t][:, :, None] * S + kv
    return torch.stack(out), S


def wkv(w, p, h, m, eps):
    T = h.shape[0]
    H, D = m["heads"], m["dim"]
    mix = {s: token_mix(h, w[f"{p}mu.{s}"]) for s in "rkvgw"}
    r, k, v = ((mix[s] @ w[p + s].t()).view(T, H, D) for s in "rkv")
    gate = F.silu(mix["g"] @ w[p + "g"].t())
    decay = torch.exp(-torch.exp(torch.tanh(mix["w"] @ w[p + "w1"].t()) @ w[p + "w2"].t() + w[p + "w0"])).view(T, H, D)
    o, _ = wkv_recurrence(r, k, v, decay, w[p + "u"])
    o = rms(o, eps).reshape(T, H * D) * w[p + "norm"] * gate
    return o @ w[p + "o"].t()


# ---------------------------------------------------------------------------------------------- windowed attention
def frequencies(rot):
    """Angle per position of every rotated pair, long wavelengths slowed down (Llama 3.1 rule) when `scaling` is given."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        s = rot.get("scaling")
        if s:
            wavelength = 2 * math.pi / f
            if wavelength > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wavelength >= s["original"] / s["high"]:
                t = (s["original"] / wavelength - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return torch.tensor(out, dtype=torch.float64)


def rotate_half(x, positions, rot):
    """x [T, heads, d]: of the first `dims` coordinates, i turns with i + dims/2."""
    n = rot["dims"]
    ang = positions.to(torch.float64)[:, None] * frequencies(rot)
    c, s = ang.cos().to(x.dtype)[:, None], ang.sin().to(x.dtype)[:, None]
    u, v = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., n:]], dim=-1)


def window_mask(n, size):
    i = torch.arange(n)
    d = i[:, None] - i[None, :]
    return (d >= 0) & (d < size)


def window_attention(w, p, h, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    pos = torch.arange(T)
    q = (h @ w[p + "q"].t()).view(T, H, D)
    k = (h @ w[p + "k"].t()).view(T, G, D)
    v = (h @ w[p + "v"].t()).view(T, G, V)
    q = rotate_half(rms(q, eps) * w[p + "q.norm"], pos, m["rot"])
    k = rotate_half(rms(k, eps) * w[p + "k.norm"], pos, m["rot"])
    out = []
    for i in range(H):
        g = i // (H // G)
        s = (q[:, i] @ k[:, g].t()) * m["scale"]
        s = s.masked_fill(~window_mask(T, m["mask"]["size"]), float("-inf"))
        out.append(torch.softmax(s, dim=-1) @ v[:, g])
    return torch.cat(out, dim=-1) @ w[p + "o"].t()


# ---------------------------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """x [T, C], taps [C, n] (last: the current token): causal convolution per channel, then silu."""
    n = taps.shape[1]
    padded = torch.cat([torch.zeros(n - 1, x.shape[1], dtype=x.dtype), x])
    return F.silu(sum(padded[j:j + x.shape[0]] * taps[:, j] for j in range(n)))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_recurrence(q, k, v, decay, beta, state=None):
    """q, k [T, H, D], v [T, H, V], decay, beta [T, H] -> o [T, H, V] and the last state [H, D, V]."""
    T, H, D = q.shape
    S = torch.zeros(H, D, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hdv,hd->hv", S, q[t]))
    return torch.stack(out), S


def gated_delta(w, p, h, m, eps):
    T = h.shape[0]
    H, G, D, V = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w[p + "q"].t(), w[p + "q.conv"]).view(T, G, D)
    k = short_conv(h @ w[p + "k"].t(), w[p + "k.conv"]).view(T, G, D)
    v = short_conv(h @ w[p + "v"].t(), w[p + "v.conv"]).view(T, H, V)
    q, k = unit(q) * D ** -0.5, unit(k)
    group = torch.arange(H) // (H // G)
    beta = torch.sigmoid(h @ w[p + "b"].t())
    decay = torch.exp(-torch.exp(w[p + "A_log"]) * F.softplus(h @ w[p + "a"].t() + w[p + "dt_bias"]))
    o, _ = delta_recurrence(q[:, group], k[:, group], v, decay, beta)
    gate = F.silu(h @ w[p + "g"].t()).view(T, H, V)
    return (rms(o, eps) * w[p + "norm"] * gate).reshape(T, H * V) @ w[p + "o"].t()


def parallel(w, p, h, m, eps):
    return m["left_scale"] * window_attention(w, p + "left.", h, m["left"], eps) + \
        m["right_scale"] * gated_delta(w, p + "right.", h, m["right"], eps)


# ---------------------------------------------------------------------------------------------- the rest
def feed_forward(w, p, h):
    return torch.relu(h @ w[p + "up"].t()).square() @ w[p + "down"].t()


MIXERS = {"wkv": wkv, "parallel": parallel}


def layers(w, cfg, tokens):
    """Residual stream after every layer [L, T, width]."""
    eps = cfg["norm"]["eps"]
    x, out = embed(w, tokens, cfg), []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + norm1p(MIXERS[layer["type"]](w, p + "mix.", x, layer["mixer"], eps), w[p + "norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + norm1p(feed_forward(w, p + "mlp.", x), w[p + "norm2"], eps)
        out.append(x)
    return torch.stack(out)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def logits(w, cfg, tokens):
    """Logits of every position [T, vocab]."""
    x = norm1p(layers(w, cfg, tokens)[-1], w["final.norm"], cfg["norm"]["eps"])
    return softcap(x @ w["embed"].t(), cfg["logit_softcap"])


def greedy(w, cfg, tokens, n):
    ids = list(tokens)
    for _ in range(n):
        ids.append(int(logits(w, cfg, ids)[-1].argmax()))
    return ids[len(tokens):]


# ---------------------------------------------------------------------------------------------- test models
def at(v, i):
    """Value of layer i: lists hold one value per layer (repeated)."""
    return v[i % len(v)] if isinstance(v, (list, tuple)) else v


SCALING = {"factor": 3.0, "low": 1.0, "high": 3.5, "original": 90}


def make_config(width=64, vocab=300, types=("parallel", "wkv", "parallel"), heads=4, kv_heads=2, dim=16, vdim=24, window=7, rot=8,
                base=500.0, scaling=SCALING, scale=None, dheads=4, dkv=2, ddim=16, dvdim=24, taps=3, left_scale=0.8,
                right_scale=1.3, wheads=3, wdim=16, ff=80, embed_scale=2.5, softcap=20.0, eps=1e-5, decay_rank=12, mlp_every=1):
    """A configuration dictionary as a checkpoint's config.json holds it.  Sizes may be lists (one value per layer);
    `mlp_every` > 1 leaves layers without a feed-forward in between."""
    ls = []
    for i, kind in enumerate(types):
        if kind == "wkv":
            mixer = {"heads": at(wheads, i), "dim": at(wdim, i), "decay_rank": at(decay_rank, i)}
        else:
            d, sc = at(dim, i), at(scaling, i)
            r = {"base": at(base, i), "dims": at(rot, i)}
            if sc:
                r["scaling"] = dict(sc)
            mixer = {"left": {"heads": at(heads, i), "kv_heads": at(kv_heads, i), "dim": d, "vdim": at(vdim, i),
                              "mask": {"size": at(window, i)}, "rot": r,
                              "scale": at(scale, i) if scale is not None else d ** -0.5},
                     "right": {"heads": at(dheads, i), "kv_heads": at(dkv, i), "dim": at(ddim, i), "vdim": at(dvdim, i),
                               "conv": at(taps, i)},
                     "left_scale": at(left_scale, i), "right_scale": at(right_scale, i)}
        ls.append({"type": kind, "mixer": mixer, "mlp": {"kind": "dense", "ff": at(ff, i)} if i % mlp_every == 0 else None})
    return {"architecture": "Vibepel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "logit_softcap": softcap, "layers": ls}


def make_weights(cfg, seed=0, sharp=1.0, slow=False):
    """Random weights (bf16-representable float32).  `sharp` scales the norm weights of queries and keys, so that a wrong key
    changes the outcome instead of drowning in an even average; `slow` lets recurrent states remember for long."""
    g = torch.Generator().manual_seed(seed)
    W = cfg["width"]

    def lin(o, i, s=1.0):
        return torch.randn(o, i, generator=g) * (s / math.sqrt(i))

    def near(n, c, s=0.2):
        return c + s * torch.randn(n, generator=g)

    w = {"embed": torch.randn(cfg["vocab"], W, generator=g) / math.sqrt(W) * 2}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], f"l{i}.mix."
        w[f"l{i}.norm1"] = near(W, 0.0)
        if layer["type"] == "wkv":
            n = m["heads"] * m["dim"]
            for s in "rkvgw":
                w[p + "mu." + s] = torch.rand(W, generator=g)
            for s in "rkvg":
                w[p + s] = lin(n, W)
            w[p + "w1"], w[p + "w2"] = lin(m["decay_rank"], W), lin(n, m["decay_rank"], 2.0)
            w[p + "w0"] = near(n, -5.0 if slow else -1.5, 1.0)
            w[p + "u"], w[p + "norm"], w[p + "o"] = near((m["heads"], m["dim"]), 0.5, 0.5), near(n, 1.0), lin(W, n)
        else:
            a, b = m["left"], m["right"]
            H, G, D, V = a["heads"], a["kv_heads"], a["dim"], a["vdim"]
            w[p + "left.q"], w[p + "left.k"], w[p + "left.v"] = lin(H * D, W), lin(G * D, W), lin(G * V, W)
            w[p + "left.q.norm"], w[p + "left.k.norm"] = near(D, sharp), near(D, sharp)
            w[p + "left.o"] = lin(W, H * V)
            H, G, D, V = b["heads"], b["kv_heads"], b["dim"], b["vdim"]
            for s, n in (("q", G * D), ("k", G * D), ("v", H * V)):
                w[p + "right." + s] = lin(n, W)
                w[p + f"right.{s}.conv"] = torch.randn(n, b["conv"], generator=g) * 0.7
            w[p + "right.b"], w[p + "right.a"], w[p + "right.g"] = lin(H, W), lin(H, W), lin(H * V, W)
            w[p + "right.A_log"] = near(H, 0.0, 0.5)
            w[p + "right.dt_bias"] = near(H, -5.0 if slow else -1.0, 0.5)
            w[p + "right.norm"], w[p + "right.o"] = near(V, 1.0), lin(W, H * V)
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            w[f"l{i}.norm2"] = near(W, 0.0)
            w[f"l{i}.mlp.up"], w[f"l{i}.mlp.down"] = lin(ff, W), lin(W, ff)
    w["final.norm"] = near(W, 0.5)
    return {k: v.to(torch.bfloat16).float() for k, v in w.items()}
