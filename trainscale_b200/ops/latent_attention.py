"""Latent attention: a compressed key/value row per token shared by all heads (csrc/latent.cu, csrc/latent_prefill.cu).

Two forms of the same attention:
  * in latent space (`attend_latent`): the query is carried into the latent space of the cache, scores and the weighted
    sum use the cached rows themselves.  Single query rows - decoding, fp32, and head sizes the tensor-core kernel does
    not take.
  * expanded (`attend_expanded`): per-head keys and values are rebuilt from the latents of a portion and its window by one
    GEMM, then a tcgen05 flash kernel runs over them.  Portions of prompts in bf16.
Tensors on the CPU take PyTorch math.
"""
from __future__ import annotations

import ctypes
import functools
from dataclasses import dataclass

import torch

from . import _lib
from .masks import KeyMask

_ll, _f = ctypes.c_longlong, ctypes.c_float


@dataclass(frozen=True)
class LatentShape:
    """Sizes and constants of one latent-attention layer."""
    heads: int
    dim: int              # unrotated query / key size per head
    rot: int              # rotated size per head
    vdim: int             # value size per head
    rank: int             # latent size
    window: int           # keys a position sees: itself and window - 1 before it
    scale: float
    rope_base: float = 10000.0
    pairs: bool = False   # rotation partners: coordinates 2 i and 2 i + 1 instead of i and i + rot / 2
    magnitude: float = 1.0  # factor of cos and sin

    @property
    def q_width(self) -> int:
        return self.heads * (self.dim + self.rot)

    @property
    def mask(self) -> KeyMask:
        return KeyMask(self.window)

    @property
    def row_width(self) -> int:
        """Columns of a cache row: rank + rot, padded with zeros to a multiple of 16."""
        return -(-(self.rank + self.rot) // 16) * 16


@functools.lru_cache(maxsize=None)
def expanded_supported(s: LatentShape) -> bool:
    return s.scale > 0 and s.rank % 8 == 0 and bool(_lib.load("latent_prefill").ts_latent_prefill_supported(s.dim, s.rot, s.vdim))


def _rotate(x: torch.Tensor, cos: torch.Tensor, sin: torch.Tensor, pairs: bool) -> torch.Tensor:
    if pairs:
        u, v = x[..., 0::2].float(), x[..., 1::2].float()
        return torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2).to(x.dtype)
    half = x.shape[-1] // 2
    u, v = x[..., :half].float(), x[..., half:].float()
    return torch.cat([u * cos - v * sin, v * cos + u * sin], dim=-1).to(x.dtype)


def prepare(proj: torch.Tensor, s: LatentShape, norm_w, eps: float, inv_freq, pos, slots, cache, keep_rows: bool):
    """proj [T, >= q_width + rank + rot] = (queries | latent | shared key part | ...).  Rotates the queries in place, writes the
    normed latent and the rotated key part to cache rows `slots`; returns those rows [T, row_width] if `keep_rows`."""
    T = proj.shape[0]
    if not proj.is_cuda:
        ang = pos.float()[:, None] * inv_freq
        cos, sin = ang.cos() * s.magnitude, ang.sin() * s.magnitude
        q = proj[:, :s.q_width].view(T, s.heads, s.dim + s.rot)
        q[..., s.dim:] = _rotate(q[..., s.dim:], cos[:, None], sin[:, None], s.pairs)
        c = proj[:, s.q_width:s.q_width + s.rank].float()
        rows = torch.zeros(T, s.row_width, dtype=proj.dtype)
        rows[:, :s.rank] = (c / torch.sqrt(c.pow(2).mean(-1, keepdim=True) + eps) * norm_w).to(proj.dtype)
        rows[:, s.rank:s.rank + s.rot] = _rotate(proj[:, s.q_width + s.rank:s.q_width + s.rank + s.rot], cos, sin, s.pairs)
        cache.view(-1, s.row_width)[slots] = rows
        return rows if keep_rows else None
    flat = torch.empty(T, s.row_width, dtype=proj.dtype, device=proj.device) if keep_rows else None
    rc = _lib.load("latent").ts_latent_prep(
        _lib.ptr(proj), _ll(proj.stride(0)), s.heads, s.dim, s.rot, s.rank, _lib.ptr(norm_w), _f(eps), _lib.ptr(inv_freq),
        _f(s.magnitude), int(s.pairs), _lib.ptr(pos), _lib.ptr(slots), _lib.ptr(cache), _lib.ptr(flat), s.row_width, T, int(proj.dtype == torch.float32),
        _lib.stream_ptr())
    _lib.check(rc, "ts_latent_prep")
    return flat


def gate_args(gate: torch.Tensor | None, heads: int, vdim: int, like: torch.Tensor):
    """Kernel arguments (pointer, row stride, mode) of an attention gate with one column per head or per element."""
    if gate is None:
        return _lib.ptr(None), _ll(0), 0
    if gate.dtype != like.dtype or gate.stride(1) != 1 or gate.shape[1] not in (heads, heads * vdim):
        raise ValueError("a gate has one contiguous column per head or per element, in the type of the queries")
    return _lib.ptr(gate), _ll(gate.stride(0)), 2 if gate.shape[1] == heads * vdim and vdim > 1 else 1


def gather_rows(cache: torch.Tensor, slots: torch.Tensor) -> torch.Tensor:
    """Cache rows of the given slots, contiguous."""
    w = cache.shape[-1]
    out = torch.empty(slots.numel(), w, dtype=cache.dtype, device=cache.device)
    rc = _lib.load("latent").ts_latent_gather(_lib.ptr(cache), _lib.ptr(slots), _lib.ptr(out), _ll(slots.numel()),
                                              w * cache.element_size(), _lib.stream_ptr())
    _lib.check(rc, "ts_latent_gather")
    return out


def attend_latent(q_lat: torch.Tensor, proj: torch.Tensor, s: LatentShape, cache, block_table, row_seq, row_len,
                  max_len: int) -> torch.Tensor:
    """q_lat [T, H, rank]; proj [T, ...] with the rotated queries; row r belongs to row `row_seq[r]` of the block table
    (None: r) and sees the keys before row_len[r] inside the window.  Returns the latent sums [T, H, rank]."""
    T, H, rank = q_lat.shape
    bs = cache.shape[1]
    if not q_lat.is_cuda:
        out = torch.empty_like(q_lat)
        flat = cache.view(-1, s.row_width)
        qr = proj[:, :s.q_width].view(T, H, s.dim + s.rot)[..., s.dim:]
        for t in range(T):
            n = int(row_len[t])
            j = torch.arange(max(0, n - s.window), n)
            rows = flat[block_table[int(row_seq[t]) if row_seq is not None else t][j // bs].long() * bs + j % bs]
            sc = (q_lat[t] @ rows[:, :rank].t() + qr[t] @ rows[:, rank:rank + s.rot].t()).float() * s.scale
            out[t] = torch.softmax(sc, -1).to(q_lat.dtype) @ rows[:, :rank]
        return out
    lib = _lib.load("latent")
    fp32 = int(q_lat.dtype == torch.float32)
    keys = min(s.window, max_len)
    splits = lib.ts_latent_splits(T, H, rank, s.row_width, bs, keys, fp32)
    out = torch.empty_like(q_lat)
    po = pl = None
    if splits > 1:
        po = torch.empty(T, H, splits, rank, dtype=torch.float32, device=q_lat.device)
        pl = torch.empty(T, H, splits, dtype=torch.float32, device=q_lat.device)
    rc = lib.ts_latent_attend(_lib.ptr(q_lat), _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(cache), _lib.ptr(block_table),
                              block_table.shape[1], _lib.ptr(row_seq), _lib.ptr(row_len), _lib.ptr(out), _lib.ptr(po),
                              _lib.ptr(pl), T, H, s.dim, s.rot, rank, s.row_width, bs, s.window, keys, splits, _f(s.scale),
                              fp32, _lib.stream_ptr())
    _lib.check(rc, "ts_latent_attend")
    return out


def attend_expanded(proj: torch.Tensor, kv: torch.Tensor, rows: torch.Tensor, s: LatentShape, cu_q, cu_k, max_q: int,
                    out: torch.Tensor, gate: torch.Tensor | None = None) -> None:
    """proj [Tq, ...] with the queries; kv [Tk, H * dim + H * vdim] expanded keys | values of the latent rows `rows`
    [Tk, row_width]; cu_q / cu_k int32 offsets of every sequence (its queries are the last of its keys).  Writes
    out [Tq, H * vdim], times sigmoid(gate) when there is a gate [Tq, H * vdim] or (one per head) [Tq, H]."""
    gp, gld, mode = gate_args(gate, s.heads, s.vdim, proj)
    rc = _lib.load("latent_prefill").ts_latent_prefill(
        _lib.ptr(proj), _ll(proj.stride(0)), _ll(proj.shape[0]), _lib.ptr(kv), _ll(kv.stride(0)), s.heads * s.dim,
        ctypes.c_void_p(rows.data_ptr() + s.rank * rows.element_size()), _ll(rows.stride(0)), _ll(rows.shape[0]),
        _lib.ptr(cu_q), _lib.ptr(cu_k), cu_q.numel() - 1, max_q, s.heads, s.dim, s.rot, s.vdim, s.window, _f(s.scale),
        gp, gld, mode, _lib.ptr(out), _ll(out.stride(0)), _lib.stream_ptr())
    _lib.check(rc, "ts_latent_prefill")
