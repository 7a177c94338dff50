"""Attention with grouped queries over a part of the keys (csrc/window.cu, csrc/latent_prefill.cu): a sliding window, with or
without the sequence's first positions, chunks, or all of them (`masks.UNBOUNDED`).  Optional bias, per-head RMS norm of queries and
keys, a factor of the queries that grows with the position, rotary embedding of part of a head, a gate on the result; keys and
values of unlike sizes side by side in one paged cache row per token.  Weights are a softmax of the scores or their sigmoids;
scores may carry a number per head and a slope per head over the distance (`ScoreBias`).

`attend_rows` serves single query rows (decoding, fp32, sizes the tensor-core prefill kernel does not take),
`attend_portions` portions of prompts in bf16.  Tensors on the CPU take PyTorch math.
"""
from __future__ import annotations

import ctypes
import functools
import math
from dataclasses import dataclass

import torch

from . import _lib
from .latent_attention import gate_args
from .masks import UNBOUNDED, KeyMask

_ll, _f = ctypes.c_longlong, ctypes.c_float


@dataclass(frozen=True)
class WindowShape:
    """Sizes and constants of one attention mixer."""
    heads: int
    kv_heads: int
    dim: int              # query / key size per head
    vdim: int             # value size per head
    rot: int              # rotated dimensions of a head
    window: int           # keys a position sees (`mask`)
    scale: float
    keep: int = 0
    chunked: bool = False
    pairs: bool = False   # rotation partners: coordinates 2 i and 2 i + 1 instead of i and i + rot / 2
    values_are_keys: bool = False   # values are the keys as projected, before norm and rotation
    sigmoid: bool = False           # weights are sigmoids of the scores, not normalized over keys
    temperature: tuple[float, int] | None = None   # (coef, every): queries times 1 + coef ln(floor((p + 1) / every) + 1)

    @property
    def mask(self) -> KeyMask:
        return KeyMask(self.window, self.keep, self.chunked)

    @property
    def q_width(self) -> int:
        return self.heads * self.dim

    @property
    def in_width(self) -> int:
        """Columns that are projected: queries, keys and (unless they are the keys) values."""
        return self.q_width + self.kv_heads * (self.dim + (0 if self.values_are_keys else self.vdim))

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


@dataclass
class ScoreBias:
    """Terms of a head's scores besides q . k * scale, fp32 [heads]; either may be None."""
    slopes: torch.Tensor | None = None    # times the distance of query and key, taken off
    add: torch.Tensor | None = None
    limit: float = math.inf               # no q . k * scale exceeds it; then sigmoid weights that fade with the distance are left
                                          # out where they are below 2^-48


NO_BIAS = ScoreBias()


def distance_slopes(heads: int) -> torch.Tensor:
    """Slopes 2^(-8 (h + 1) / heads), a geometric series over the heads that ends at 2^-8."""
    return torch.tensor([2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)], dtype=torch.float32)


def sigmoid_reach(limit: float, add: float, slope: float) -> int:
    """Distance up to which a sigmoid weight can be 2^-48 or more, as the kernels compute it."""
    return UNBOUNDED if math.isinf(limit) or slope <= 0 else max(0, min(UNBOUNDED, int((limit + add + 33.28) / slope) + 1))


@functools.lru_cache(maxsize=None)
def portions_supported(s: WindowShape) -> bool:
    """Whether `attend_portions` takes these sizes (a bias of the scores: only with sigmoid weights)."""
    return s.scale > 0 and bool(_lib.load("latent_prefill").ts_latent_prefill_supported(s.dim, 0, s.vdim))


def _norm_rotate(y: torch.Tensor, w, eps: float, cs: torch.Tensor | None, s: WindowShape) -> torch.Tensor:
    if w is not None:
        y = y / torch.sqrt(y.pow(2).mean(-1, keepdim=True) + eps) * w
    if not s.rot:
        return y
    cos, sin = cs[:, None, :s.rot // 2], cs[:, None, s.rot // 2:]
    if s.pairs:
        u, v = y[..., 0:s.rot:2], y[..., 1:s.rot:2]
        turned = torch.stack([u * cos - v * sin, v * cos + u * sin], dim=-1).flatten(-2)
    else:
        u, v = y[..., :s.rot // 2], y[..., s.rot // 2:s.rot]
        turned = torch.cat([u * cos - v * sin, v * cos + u * sin], dim=-1)
    return torch.cat([turned, y[..., s.rot:]], dim=-1)


def angles(inv_freq: torch.Tensor, pos: torch.Tensor, magnitude: float = 1.0) -> torch.Tensor:
    """cos | sin of pos * inv_freq, times `magnitude`, fp32 [T, 2 * frequencies]: once per step for all layers that rotate
    alike."""
    if not pos.is_cuda:
        a = pos.float()[:, None] * inv_freq
        return torch.cat([a.cos(), a.sin()], dim=-1) * magnitude
    out = torch.empty(pos.shape[0], 2 * inv_freq.shape[0], dtype=torch.float32, device=pos.device)
    rc = _lib.load("window").ts_window_angles(_lib.ptr(inv_freq), _lib.ptr(pos), _lib.ptr(out), pos.shape[0], inv_freq.shape[0],
                                              _f(magnitude), _lib.stream_ptr())
    _lib.check(rc, "ts_window_angles")
    return out


def prepare(proj: torch.Tensor, s: WindowShape, q_norm, k_norm, eps: float, cs: torch.Tensor | None, slots, cache,
            bias: torch.Tensor | None = None, pos: torch.Tensor | None = None) -> None:
    """proj [T, >= q_width + kv_width] = (queries | keys | values | ...); cs of `angles`; norms and bias (fp32, of queries and
    keys) may be None; pos int32 [T] for shapes with a temperature.  Norms and rotates queries and keys in place and writes keys and values to cache rows `slots`; the
    value columns of proj are written when the values are the keys."""
    T = proj.shape[0]
    if not proj.is_cuda:
        kw = s.kv_heads * s.dim
        qk = proj[:, :s.q_width + kw].to(torch.float32, copy=True)
        if bias is not None:
            qk = qk + bias
        if s.values_are_keys:
            proj[:, s.q_width + kw:s.q_width + s.kv_width] = qk[:, s.q_width:]
        q, k = qk[:, :s.q_width].view(T, s.heads, s.dim), qk[:, s.q_width:].view(T, s.kv_heads, s.dim)
        q = _norm_rotate(q, q_norm, eps, cs, s)
        if s.temperature is not None:
            coef, every = s.temperature
            q = q * (1 + coef * torch.log((pos + 1).div(every, rounding_mode="floor") + 1.0))[:, None, None]
        proj[:, :s.q_width] = q.reshape(T, -1)
        proj[:, s.q_width:s.q_width + kw] = _norm_rotate(k, k_norm, eps, cs, s).reshape(T, -1)
        cache.view(-1, s.row_width)[slots, :s.kv_width] = proj[:, s.q_width:s.q_width + s.kv_width]
        return
    coef, every = s.temperature or (0.0, 0)
    rc = _lib.load("window").ts_window_prep(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(bias), _lib.ptr(q_norm), _lib.ptr(k_norm), _f(eps), _lib.ptr(cs),
        _lib.ptr(slots), _lib.ptr(cache), T, s.heads, s.kv_heads, s.dim, s.vdim, s.rot, int(s.pairs), int(s.values_are_keys),
        _lib.ptr(pos if every else None), _f(coef), every, s.row_width, int(proj.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_window_prep")


def attend_rows(proj: torch.Tensor, s: WindowShape, cache, block_table, row_seq, row_len, max_len: int, out: torch.Tensor,
                out_scale: float = 1.0, gate: torch.Tensor | None = None, bias: ScoreBias = NO_BIAS) -> None:
    """out [T, out_width] = out_scale * attention of the query rows proj[:, :q_width]; row r belongs to row `row_seq[r]` of
    the block table and sees the keys before row_len[r] that the mask leaves.  `gate` ([T, heads] or [T, out_width]): the
    result is multiplied by its sigmoid."""
    T, bs = proj.shape[0], cache.shape[1]
    if not proj.is_cuda:
        flat = cache.view(-1, s.row_width)
        kw = s.kv_heads * s.dim
        for t in range(T):
            j = torch.tensor(s.mask.positions(int(row_len[t]) - 1))
            rows = flat[block_table[int(row_seq[t])][j // bs].long() * bs + j % bs].float()
            q = proj[t, :s.q_width].float().view(s.kv_heads, -1, s.dim)
            k = rows[:, :kw].view(-1, s.kv_heads, s.dim)
            v = rows[:, kw:s.kv_width].view(-1, s.kv_heads, s.vdim)
            sc = torch.einsum("ghd,jgd->ghj", q, k) * s.scale
            if bias.slopes is not None:
                sc = sc - bias.slopes.view(s.kv_heads, -1, 1) * (int(row_len[t]) - 1 - j).float()
            if bias.add is not None:
                sc = sc + bias.add.view(s.kv_heads, -1, 1)
            w = torch.sigmoid(sc) if s.sigmoid else torch.softmax(sc, -1)
            o = (torch.einsum("ghj,jgv->ghv", w, v) * out_scale).reshape(s.heads, s.vdim)
            if gate is not None:
                o = o * torch.sigmoid(gate[t].float()).view(s.heads, -1)
            out[t] = o.reshape(-1).to(out.dtype)
        return
    gp, gld, mode = gate_args(gate, s.heads, s.vdim, proj)
    lib = _lib.load("window")
    fp32 = int(proj.dtype == torch.float32)
    keys = s.mask.most(max_len)
    splits = lib.ts_window_splits(T, s.heads, s.kv_heads, s.dim, s.vdim, keys, fp32)
    po = pl = None
    if splits > 1:
        po = torch.empty(T, s.heads, splits, s.vdim, dtype=torch.float32, device=proj.device)
        pl = torch.empty(T, s.heads, splits, dtype=torch.float32, device=proj.device)
    rc = lib.ts_window_attend(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(cache), _lib.ptr(block_table), block_table.shape[1], _lib.ptr(row_seq),
        _lib.ptr(row_len), _lib.ptr(out), _ll(out.stride(0)), _lib.ptr(po), _lib.ptr(pl), T, s.heads, s.kv_heads, s.dim,
        s.vdim, s.row_width, bs, s.window, s.keep, int(s.chunked), keys, splits, _f(s.scale), _f(out_scale), _lib.ptr(bias.slopes),
        _lib.ptr(bias.add), int(s.sigmoid), _f(bias.limit), gp, gld, mode, fp32, _lib.stream_ptr())
    _lib.check(rc, "ts_window_attend")


def attend_portions(proj: torch.Tensor, s: WindowShape, rows: torch.Tensor | None, cu_q, cu_k, max_q: int, out: torch.Tensor,
                    out_scale: float = 1.0, gate: torch.Tensor | None = None, bias: ScoreBias = NO_BIAS) -> None:
    """Portions of prompts, bf16: queries proj[:, :q_width]; keys and values of every sequence, in key order, in `rows`
    [Tk, row_width] (None: exactly the portions' own, beside the queries).  cu_q / cu_k int32 offsets of every sequence
    (its queries are the last of its keys): the kept first positions, if they are not part of the window's run, then the
    positions from the first query's window or chunk on."""
    gp, gld, mode = gate_args(gate, s.heads, s.vdim, proj)
    at = proj.data_ptr() + s.q_width * proj.element_size() if rows is None else rows.data_ptr()
    src = proj if rows is None else rows
    rc = _lib.load("latent_prefill").ts_window_prefill(
        _lib.ptr(proj), _ll(proj.stride(0)), _ll(proj.shape[0]), ctypes.c_void_p(at),
        ctypes.c_void_p(at + s.kv_heads * s.dim * proj.element_size()), _ll(src.stride(0)), _ll(src.shape[0]), _lib.ptr(cu_q),
        _lib.ptr(cu_k), cu_q.numel() - 1, max_q, s.heads, s.kv_heads, s.dim, s.vdim, s.window, s.keep, int(s.chunked),
        _f(s.scale), _f(out_scale), _lib.ptr(bias.slopes), _lib.ptr(bias.add), int(s.sigmoid), _f(bias.limit), gp, gld, mode,
        _lib.ptr(out), _ll(out.stride(0)), _lib.stream_ptr())
    _lib.check(rc, "ts_window_prefill")
