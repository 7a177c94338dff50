"""Residual-stream boundary ops of decoders with an fp32 stream (csrc/stream.cu).

Depth-averaged stream: `embed` starts it (token row + bigram row), `boundary` closes one layer and opens the next: residual sum of a
parallel block, expert combine, depth average over every earlier result, scalar-gain RMS norm and token shift in one
launch; `final` is the last boundary for the rows whose logits are wanted.  Output-normed sublayers: `scaled_embed`,
`postnorm` (sum, cast or token-shift mixes) and `postnorm_final`.  Input-normed sublayers: `prenorm_embed`, `prenorm` (sum
with a gated addend and an expert combine, norm) and `prenorm_final`.  The stream, its history and the per-sequence
state are fp32; h and hs come out in the activation dtype.  Tensors on the CPU take PyTorch math.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib

_ll, _f = ctypes.c_longlong, ctypes.c_float
ROW_BEFORE = -2      # row_prev: the previous row of the batch
ROW_ZERO = -1        # row_prev: no previous token


@dataclass
class StreamRows:
    """Where every row of the batch finds the row before it, and which rows leave their h behind."""
    prev: torch.Tensor        # [T] int32: state row, ROW_ZERO or ROW_BEFORE
    next: torch.Tensor        # [T] int32: state row that receives h, or -1


def _fp32(t: torch.Tensor) -> int:
    if t.dtype not in (torch.float32, torch.bfloat16):
        raise TypeError(f"stream kernels take float32 or bfloat16 activations, not {t.dtype}")
    return int(t.dtype == torch.float32)


def scalar_rmsnorm(x: torch.Tensor, gain: torch.Tensor, eps: float) -> torch.Tensor:
    return x * (gain / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps))


def _shift(h: torch.Tensor, shift: torch.Tensor, rows: StreamRows, state: torch.Tensor) -> torch.Tensor:
    prev = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    p = rows.prev.long()
    prev = torch.where((p >= 0)[:, None], state[p.clamp(min=0)], prev)
    prev = torch.where((p == ROW_ZERO)[:, None], torch.zeros_like(prev), prev)
    hs = h + (prev - h) * shift
    n = rows.next.long()
    state[n[n >= 0]] = h[n >= 0]
    return hs


def embed(tok, prev_tok, table, bigram, mul_prev: int, mul_cur: int, hist, gain, eps: float, shift, rows: StreamRows,
          state) -> tuple[torch.Tensor, torch.Tensor]:
    """X_0 -> hist[0]; returns (h, hs) of the first layer."""
    T, W = tok.shape[0], table.shape[1]
    buckets = bigram.shape[0] - 1
    if not tok.is_cuda:
        p = prev_tok.long()
        row = torch.where(p < 0, torch.full_like(p, buckets), (p.clamp(min=0) * mul_prev + tok.long() * mul_cur) % buckets)
        x = table[tok.long()].float() + bigram[row].float()
        hist[0, :T] = x
        h = scalar_rmsnorm(x, gain, eps)
        return h.to(table.dtype), _shift(h, shift, rows, state).to(table.dtype)
    h, hs = (torch.empty(T, W, dtype=table.dtype, device=tok.device) for _ in range(2))
    rc = _lib.load("stream").ts_stream_embed(
        _lib.ptr(tok), _lib.ptr(prev_tok), _lib.ptr(table), _lib.ptr(bigram), table.shape[0], buckets, _ll(mul_prev),
        _ll(mul_cur), _lib.ptr(hist), _lib.ptr(gain), _f(eps), _lib.ptr(shift), _lib.ptr(h), _lib.ptr(hs),
        _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(state), T, W, _fp32(table), _lib.stream_ptr())
    _lib.check(rc, "ts_stream_embed")
    return h, hs


def _sum(x, mixer, experts, hist, dwa, n):
    v = x.clone()
    if mixer is not None:
        v = v + mixer.float()
    if experts is not None:
        y, dest, w = experts
        T, k = w.shape
        idx = dest.long().view(T, k) if dest is not None else torch.arange(T * k).view(T, k)
        v = v + (y[idx].float() * w.unsqueeze(-1)).sum(1)
    avg = dwa[n] * v
    for j in range(n):
        avg = avg + dwa[j] * hist[j, :v.shape[0]]
    return v, avg


def _boundary_raw(x, mixer, experts, hist, dwa, n, x_out, gain, eps, shift, h, hs, rows, state, out_rows):
    y, dest, w = experts if experts is not None else (None, None, None)
    T, W = x.shape
    rc = _lib.load("stream").ts_stream_layer(
        _lib.ptr(x), _lib.ptr(mixer), 0 if mixer is None else mixer.stride(0), _lib.ptr(y), _lib.ptr(dest), _lib.ptr(w),
        0 if w is None else w.shape[1], _lib.ptr(hist), _ll(hist.stride(0)), _lib.ptr(dwa), n, _lib.ptr(x_out),
        _lib.ptr(gain), _f(eps), _lib.ptr(shift), _lib.ptr(h), _lib.ptr(hs), _lib.ptr(None if rows is None else rows.prev),
        _lib.ptr(None if rows is None else rows.next), _lib.ptr(state), T, _lib.ptr(out_rows),
        0 if out_rows is None else out_rows.numel(), W, _fp32(h), _lib.stream_ptr())
    _lib.check(rc, "ts_stream_layer")


def boundary(x, mixer, experts, hist, dwa, n: int, gain, eps: float, shift, rows: StreamRows, state, act_dtype):
    """x [T, W] fp32 stream; mixer [T, W]; experts = (outputs, dest or None, weights [T, k]) or None; hist
    [layers + 1, T, W] holds n results, the n-th is written.  Returns (x', h, hs); x' is a new tensor."""
    if not x.is_cuda:
        v, avg = _sum(x, mixer, experts, hist, dwa, n)
        hist[n, :x.shape[0]] = v
        h = scalar_rmsnorm(avg, gain, eps)
        return avg, h.to(act_dtype), _shift(h, shift, rows, state).to(act_dtype)
    x_out = torch.empty_like(x)
    h, hs = (torch.empty(x.shape, dtype=act_dtype, device=x.device) for _ in range(2))
    _boundary_raw(x, mixer, experts, hist, dwa, n, x_out, gain, eps, shift, h, hs, rows, state, None)
    return x_out, h, hs


def final(x, mixer, experts, hist, dwa, n: int, gain, eps: float, out_rows, act_dtype) -> torch.Tensor:
    """Normed result of the last layer for the rows `out_rows` (int32)."""
    if not x.is_cuda:
        _, avg = _sum(x, mixer, experts, hist, dwa, n)
        return scalar_rmsnorm(avg[out_rows.long()], gain, eps).to(act_dtype)
    h = torch.empty(out_rows.numel(), x.shape[1], dtype=act_dtype, device=x.device)
    if out_rows.numel():
        _boundary_raw(x, mixer, experts, hist, dwa, n, None, gain, eps, None, h, None, None, None, out_rows)
    return h


# ---------------------------------------------------------------------------------------------- output-normed boundaries
def offset_rmsnorm(x: torch.Tensor, w: torch.Tensor, eps: float) -> torch.Tensor:
    """x / rms(x) * (1 + w)."""
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (1 + w)


def _mixes(x: torch.Tensor, mu: torch.Tensor, rows: StreamRows, state: torch.Tensor) -> torch.Tensor:
    W = x.shape[1]
    prev = torch.cat([torch.zeros_like(x[:1]), x[:-1]])
    p, n = rows.prev.long(), rows.next.long()
    prev = torch.where((p >= 0)[:, None], state[p.clamp(min=0), :W], prev)
    prev = torch.where((p == ROW_ZERO)[:, None], torch.zeros_like(prev), prev)
    state[n[n >= 0], :W] = x[n >= 0]
    return x[:, None] + (prev - x)[:, None] * mu


def _postnorm_raw(tok, table, scale, x, y, w, eps, x_out, h, mu, rows, state):
    T, W = x_out.shape
    n_mix = 0 if mu is None else mu.shape[0]
    rc = _lib.load("stream").ts_stream_postnorm(
        _lib.ptr(tok), _lib.ptr(table), 0 if table is None else table.shape[0], _f(scale), _lib.ptr(x), _lib.ptr(y),
        _ll(0 if y is None else y.stride(0)), _lib.ptr(w), _f(eps), _lib.ptr(x_out), _lib.ptr(h), _lib.ptr(mu), n_mix,
        _lib.ptr(rows.prev if n_mix else None), _lib.ptr(rows.next if n_mix else None), _lib.ptr(state if n_mix else None),
        _ll(state.stride(0) if n_mix else 0), T, W, _fp32(h), _lib.stream_ptr())
    _lib.check(rc, "ts_stream_postnorm")


def _postnorm_outputs(T: int, W: int, mu, dtype, device):
    shape = (T, W) if mu is None else (T, mu.shape[0], W)
    return torch.empty(T, W, dtype=torch.float32, device=device), torch.empty(shape, dtype=dtype, device=device)


def scaled_embed(tok, table, scale: float, mu, rows: StreamRows, state):
    """x = table[tok] * scale (fp32).  Returns (x, h): h is x in the table's dtype [T, W], or with `mu` [n, W] the token-shift
    mixes x + (x of the token before - x) * mu_s [T, n, W]; `state` [rows, >= W] keeps a sequence's last x."""
    T, W = tok.shape[0], table.shape[1]
    if not tok.is_cuda:
        x = table[tok.long()].float() * scale
        return x, (x if mu is None else _mixes(x, mu, rows, state)).to(table.dtype)
    x, h = _postnorm_outputs(T, W, mu, table.dtype, tok.device)
    _postnorm_raw(tok, table, scale, None, None, None, 0.0, x, h, mu, rows, state)
    return x, h


def postnorm(x, y, w, eps: float, mu, rows: StreamRows, state, act_dtype):
    """x' = x + y / rms(y) * (1 + w) with y [T, W] the sublayer's output; returns (x', h) as `scaled_embed` does."""
    if not x.is_cuda:
        x = x + offset_rmsnorm(y.float(), w, eps)
        return x, (x if mu is None else _mixes(x, mu, rows, state)).to(act_dtype)
    x_out, h = _postnorm_outputs(*x.shape, mu, act_dtype, x.device)
    _postnorm_raw(None, None, 0.0, x, y, w, eps, x_out, h, mu, rows, state)
    return x_out, h


def postnorm_final(x, y, w, final_w, eps: float, out_rows, act_dtype) -> torch.Tensor:
    """Final norm (weight around zero) of x + y / rms(y) * (1 + w) for the rows `out_rows` (int32)."""
    if not x.is_cuda:
        r = out_rows.long()
        return offset_rmsnorm(x[r] + offset_rmsnorm(y[r].float(), w, eps), final_w, eps).to(act_dtype)
    h = torch.empty(out_rows.numel(), x.shape[1], dtype=act_dtype, device=x.device)
    rc = _lib.load("stream").ts_stream_postnorm_final(
        _lib.ptr(x), _lib.ptr(y), _ll(y.stride(0)), _lib.ptr(w), _lib.ptr(final_w), _f(eps), _lib.ptr(h), _lib.ptr(out_rows),
        out_rows.numel(), x.shape[1], _fp32(h), _lib.stream_ptr())
    _lib.check(rc, "ts_stream_postnorm_final")
    return h


# ---------------------------------------------------------------------------------------------- input-normed boundaries
@dataclass
class ElementGate:
    """Factor sigmoid(logits + bias) of every element of an addend."""
    logits: torch.Tensor      # [T, W], activation dtype
    bias: torch.Tensor        # [W] fp32


def _prenorm_norm(x, w, eps, base):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps) * (base + w)


def _prenorm_sum(x, y, y_gate, experts):
    if y is not None:
        y = y.float()
        if isinstance(y_gate, ElementGate):
            y = y * torch.sigmoid(y_gate.logits.float() + y_gate.bias)
        elif y_gate is not None:
            y = y * torch.sigmoid(y_gate)[:, None]
        x = x + y
    if experts is not None:
        e, dest, w = experts
        idx = torch.arange(w.numel()) if dest is None else dest.long()
        x = x + (e[idx].float().unflatten(0, w.shape) * w.unsqueeze(-1)).sum(1)
    return x


def _prenorm_raw(tok, table, x, y, y_gate, experts, w, base, eps, x_out, h, rows, out_rows):
    e_gate, e_bias = (y_gate.logits, y_gate.bias) if isinstance(y_gate, ElementGate) else (None, None)
    y_gate = None if e_gate is not None else y_gate
    e, dest, route_w = experts if experts is not None else (None, None, None)
    rc = _lib.load("stream").ts_stream_prenorm(
        _lib.ptr(tok), _lib.ptr(table), 0 if table is None else table.shape[0], _lib.ptr(x), _lib.ptr(y),
        _ll(0 if y is None else y.stride(0)), _lib.ptr(y_gate), _ll(0 if y_gate is None else y_gate.stride(0)),
        _lib.ptr(e_gate), _ll(0 if e_gate is None else e_gate.stride(0)), _lib.ptr(e_bias), _lib.ptr(e), _lib.ptr(dest),
        _lib.ptr(route_w), 0 if route_w is None else route_w.shape[1], _lib.ptr(w), _f(base), _f(eps), _lib.ptr(x_out),
        _lib.ptr(h), rows, _lib.ptr(out_rows), 0 if out_rows is None else out_rows.numel(), h.shape[1], _fp32(h),
        _lib.stream_ptr())
    _lib.check(rc, "ts_stream_prenorm")


def prenorm_embed(tok, table, w, eps: float, base: float = 1.0):
    """x = table[tok] (fp32); returns (x, h) with h = x / rms(x) * (base + w) in the table's dtype."""
    if not tok.is_cuda:
        x = table[tok.long()].float()
        return x, _prenorm_norm(x, w, eps, base).to(table.dtype)
    x = torch.empty(tok.shape[0], table.shape[1], dtype=torch.float32, device=tok.device)
    h = torch.empty(x.shape, dtype=table.dtype, device=tok.device)
    _prenorm_raw(tok, table, None, None, None, None, w, base, eps, x, h, tok.shape[0], None)
    return x, h


def prenorm(x, y, y_gate, experts, w, eps: float, act_dtype, base: float = 1.0):
    """x' = x + y * sigmoid(y_gate) + the weighted sum of a token's experts; returns (x', x' / rms(x') * (base + w)).
    y [T, W] or None, y_gate fp32 [T] logits, an ElementGate or None (factor one), experts of ops/moe.routed_experts or None."""
    if not x.is_cuda:
        x = _prenorm_sum(x, y, y_gate, experts)
        return x, _prenorm_norm(x, w, eps, base).to(act_dtype)
    x_out, h = torch.empty_like(x), torch.empty(x.shape, dtype=act_dtype, device=x.device)
    _prenorm_raw(None, None, x, y, y_gate, experts, w, base, eps, x_out, h, x.shape[0], None)
    return x_out, h


def prenorm_final(x, y, y_gate, experts, w, eps: float, out_rows, act_dtype, base: float = 1.0) -> torch.Tensor:
    """The norm of `prenorm` for the rows `out_rows` (int32)."""
    if not x.is_cuda:
        return _prenorm_norm(_prenorm_sum(x, y, y_gate, experts)[out_rows.long()], w, eps, base).to(act_dtype)
    h = torch.empty(out_rows.numel(), x.shape[1], dtype=act_dtype, device=x.device)
    if out_rows.numel():
        _prenorm_raw(None, None, x, y, y_gate, experts, w, base, eps, None, h, x.shape[0], out_rows)
    return h
