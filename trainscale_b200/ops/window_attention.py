"""Sliding-window attention with grouped queries (csrc/window.cu, csrc/latent_prefill.cu): per-head RMS norm of queries and
keys, rotary embedding of part of a head, keys and values of unlike sizes side by side in one paged cache row per token.

`attend_rows` serves single query rows (decoding, fp32, sizes the tensor-core prefill kernel does not take),
`attend_portions` portions of prompts in bf16.  Tensors on the CPU take PyTorch math.
"""
from __future__ import annotations

import ctypes
import functools
from dataclasses import dataclass

import torch

from . import _lib

_ll, _f = ctypes.c_longlong, ctypes.c_float


@dataclass(frozen=True)
class WindowShape:
    """Sizes and constants of one windowed-attention mixer."""
    heads: int
    kv_heads: int
    dim: int              # query / key size per head
    vdim: int             # value size per head
    rot: int              # rotated dimensions of a head
    window: int           # keys a position sees: itself and window - 1 before it
    scale: float

    @property
    def q_width(self) -> int:
        return self.heads * self.dim

    @property
    def kv_width(self) -> int:
        return self.kv_heads * (self.dim + self.vdim)

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def row_width(self) -> int:
        """Columns of a cache row: keys | values, padded with zeros to a multiple of 8."""
        return -(-self.kv_width // 8) * 8


@functools.lru_cache(maxsize=None)
def portions_supported(s: WindowShape) -> bool:
    return s.scale > 0 and bool(_lib.load("latent_prefill").ts_latent_prefill_supported(s.dim, 0, s.vdim))


def _norm_rotate(x: torch.Tensor, w: torch.Tensor, eps: float, cos: torch.Tensor, sin: torch.Tensor, rot: int) -> torch.Tensor:
    y = x.float()
    y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * w
    u, v = y[..., :rot // 2], y[..., rot // 2:rot]
    return torch.cat([u * cos - v * sin, v * cos + u * sin, y[..., rot:]], dim=-1).to(x.dtype)


def angles(inv_freq: torch.Tensor, pos: torch.Tensor) -> torch.Tensor:
    """cos | sin of pos * inv_freq, fp32 [T, 2 * frequencies]: once per step for all layers that rotate alike."""
    if not pos.is_cuda:
        a = pos.float()[:, None] * inv_freq
        return torch.cat([a.cos(), a.sin()], dim=-1)
    out = torch.empty(pos.shape[0], 2 * inv_freq.shape[0], dtype=torch.float32, device=pos.device)
    rc = _lib.load("window").ts_window_angles(_lib.ptr(inv_freq), _lib.ptr(pos), _lib.ptr(out), pos.shape[0], inv_freq.shape[0],
                                              _lib.stream_ptr())
    _lib.check(rc, "ts_window_angles")
    return out


def prepare(proj: torch.Tensor, s: WindowShape, q_norm, k_norm, eps: float, cs: torch.Tensor, slots, cache) -> None:
    """proj [T, >= q_width + kv_width] = (queries | keys | values | ...); cs of `angles`.  Norms and rotates queries and keys
    in place and writes keys and values to cache rows `slots`."""
    T = proj.shape[0]
    if not proj.is_cuda:
        cos, sin = cs[:, None, :s.rot // 2], cs[:, None, s.rot // 2:]
        q = proj[:, :s.q_width].view(T, s.heads, s.dim)
        k = proj[:, s.q_width:s.q_width + s.kv_heads * s.dim].view(T, s.kv_heads, s.dim)
        q.copy_(_norm_rotate(q, q_norm, eps, cos, sin, s.rot))
        k.copy_(_norm_rotate(k, k_norm, eps, cos, sin, s.rot))
        cache.view(-1, s.row_width)[slots, :s.kv_width] = proj[:, s.q_width:s.q_width + s.kv_width]
        return
    rc = _lib.load("window").ts_window_prep(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(q_norm), _lib.ptr(k_norm), _f(eps), _lib.ptr(cs), _lib.ptr(slots),
        _lib.ptr(cache), T, s.heads, s.kv_heads, s.dim, s.vdim, s.rot, s.row_width, int(proj.dtype == torch.float32),
        _lib.stream_ptr())
    _lib.check(rc, "ts_window_prep")


def attend_rows(proj: torch.Tensor, s: WindowShape, cache, block_table, row_seq, row_len, max_len: int, out: torch.Tensor,
                out_scale: float = 1.0) -> None:
    """out [T, out_width] = out_scale * attention of the query rows proj[:, :q_width]; row r belongs to row `row_seq[r]` of
    the block table and sees the keys before row_len[r] inside the window."""
    T, bs = proj.shape[0], cache.shape[1]
    if not proj.is_cuda:
        flat = cache.view(-1, s.row_width)
        kw = s.kv_heads * s.dim
        for t in range(T):
            n = int(row_len[t])
            j = torch.arange(max(0, n - s.window), n)
            rows = flat[block_table[int(row_seq[t])][j // bs].long() * bs + j % bs].float()
            q = proj[t, :s.q_width].float().view(s.kv_heads, -1, s.dim)
            k = rows[:, :kw].view(-1, s.kv_heads, s.dim)
            v = rows[:, kw:s.kv_width].view(-1, s.kv_heads, s.vdim)
            w = torch.softmax(torch.einsum("ghd,jgd->ghj", q, k) * s.scale, -1)
            out[t] = (torch.einsum("ghj,jgv->ghv", w, v) * out_scale).reshape(-1).to(out.dtype)
        return
    lib = _lib.load("window")
    fp32 = int(proj.dtype == torch.float32)
    keys = min(s.window, max_len)
    splits = lib.ts_window_splits(T, s.heads, s.kv_heads, s.dim, s.vdim, keys, fp32)
    po = pl = None
    if splits > 1:
        po = torch.empty(T, s.heads, splits, s.vdim, dtype=torch.float32, device=proj.device)
        pl = torch.empty(T, s.heads, splits, dtype=torch.float32, device=proj.device)
    rc = lib.ts_window_attend(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(cache), _lib.ptr(block_table), block_table.shape[1], _lib.ptr(row_seq),
        _lib.ptr(row_len), _lib.ptr(out), _ll(out.stride(0)), _lib.ptr(po), _lib.ptr(pl), T, s.heads, s.kv_heads, s.dim,
        s.vdim, s.row_width, bs, s.window, keys, splits, _f(s.scale), _f(out_scale), fp32, _lib.stream_ptr())
    _lib.check(rc, "ts_window_attend")


def attend_portions(proj: torch.Tensor, s: WindowShape, rows: torch.Tensor | None, cu_q, cu_k, max_q: int, out: torch.Tensor,
                    out_scale: float = 1.0) -> None:
    """Portions of prompts, bf16: queries proj[:, :q_width]; keys and values of every sequence, in key order, in `rows`
    [Tk, row_width] (None: exactly the portions' own, beside the queries).  cu_q / cu_k int32 offsets of every sequence
    (its queries are the last of its keys)."""
    at = proj.data_ptr() + s.q_width * proj.element_size() if rows is None else rows.data_ptr()
    src = proj if rows is None else rows
    rc = _lib.load("latent_prefill").ts_window_prefill(
        _lib.ptr(proj), _ll(proj.stride(0)), _ll(proj.shape[0]), ctypes.c_void_p(at),
        ctypes.c_void_p(at + s.kv_heads * s.dim * proj.element_size()), _ll(src.stride(0)), _ll(src.shape[0]), _lib.ptr(cu_q),
        _lib.ptr(cu_k), cu_q.numel() - 1, max_q, s.heads, s.kv_heads, s.dim, s.vdim, s.window, _f(s.scale), _f(out_scale),
        _lib.ptr(out), _ll(out.stride(0)), _lib.stream_ptr())
    _lib.check(rc, "ts_window_prefill")
