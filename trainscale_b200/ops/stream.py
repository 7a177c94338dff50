"""Residual-stream boundary ops of decoders with a depth-averaged fp32 stream (csrc/stream.cu).

`embed` starts the stream (token row + bigram row), `boundary` closes one layer and opens the next: residual sum of a
parallel block, expert combine, depth average over every earlier result, scalar-gain RMS norm and token shift in one
launch; `final` is the last boundary for the rows whose logits are wanted.  The stream, its history and the per-sequence
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
