"""Products of few rows with groups of weight matrices (csrc/skinny.cu): per-head projections, the experts of a decode
batch, and the fp32 form of both.  Tensors on the CPU take PyTorch math.

Gated products act(gate x) * (up x) have ONE weight of gate and up rows in alternating blocks (`glu_weight`): the two halves
of an output lie in the same tile of every kernel, so the product is part of the epilogue."""
from __future__ import annotations

import ctypes

import torch

from . import _lib

_ll = ctypes.c_longlong
ACT_NONE, ACT_RELU_SQUARED, ACT_TANH = 0, 1, 2
ACT_SOFTCAP, ACT_SCALE = 3, 4                # c tanh(x / c), c x; c is the constant `cap`
ACT_XIELU = 5                                # x > 0: cap x^2 + x / 2, else second (e^x - 1 - x) + x / 2
ACT_SILU_GLU, ACT_GELU_GLU = 6, 7            # silu(gate) * up, tanh form of gelu(gate) * up
ACT_BLOCK = 32                               # an activation of leading columns only takes a multiple of these
GLU_BLOCK = 16


def is_gated(act: int) -> bool:
    return act >= ACT_SILU_GLU


def glu_width(ff: int) -> int:
    """Columns of a gated product of inner size `ff`: whole blocks; those past `ff` are zero."""
    return -(-ff // GLU_BLOCK) * GLU_BLOCK


class GluRows:
    """Gate (part 0) or up (part 1) rows of a packed weight [2 * glu_width(ff), K], with the shape and copy of a plain
    [ff, K] matrix."""

    def __init__(self, packed: torch.Tensor, ff: int, part: int):
        self.blocks = packed.view(-1, 2, GLU_BLOCK, packed.shape[-1])[:, part]
        self.shape = (ff, packed.shape[-1])

    def detach(self) -> torch.Tensor:
        return self.blocks.detach().reshape(-1, self.shape[1])[:self.shape[0]]

    def copy_(self, src: torch.Tensor) -> None:
        rows = torch.zeros(self.blocks.shape[0] * GLU_BLOCK, self.shape[1], dtype=self.blocks.dtype, device=self.blocks.device)
        rows[:self.shape[0]] = src
        self.blocks.copy_(rows.view(self.blocks.shape))


def xielu(x: torch.Tensor, a: float, b: float) -> torch.Tensor:
    n = x.clamp(max=0.0)
    return a * x.clamp(min=0.0).square() + b * (torch.expm1(n) - n) + 0.5 * x


def activate(x: torch.Tensor, act: int, cap: float = 0.0, second: float = 0.0, act_cols: int | None = None) -> torch.Tensor:
    """`act` with its constants; `act_cols`: of the first columns, the others stay."""
    if act_cols is not None and act_cols < x.shape[-1]:
        return torch.cat([activate(x[..., :act_cols], act, cap, second), x[..., act_cols:]], dim=-1)
    if is_gated(act):
        g, u = x.unflatten(-1, (-1, 2, GLU_BLOCK)).unbind(-2)
        a = torch.nn.functional.silu(g) if act == ACT_SILU_GLU else torch.nn.functional.gelu(g, approximate="tanh")
        return (a * u).flatten(-2)
    if act == ACT_RELU_SQUARED:
        return torch.relu(x).square()
    if act == ACT_TANH:
        return torch.tanh(x)
    if act == ACT_SOFTCAP:
        return cap * torch.tanh(x / cap)
    if act == ACT_XIELU:
        return xielu(x, cap, second)
    return cap * x if act == ACT_SCALE else x


def _launch(A, W, out, lda, ldw, ldo, a_group, w_group, o_group, order, start, count, a_div, groups, M, N, K, act,
            typical=0, cap=0.0, gate=None, row_tiles=0, second=0.0, act_cols=None):
    if gate is not None and gate.dtype != A.dtype:
        raise TypeError("the gate has the type of the rows")
    rc = _lib.load("skinny").ts_skinny_gemm(
        _lib.ptr(A), _lib.ptr(W), _lib.ptr(out), _ll(lda), _ll(ldw), _ll(ldo), _ll(a_group), _ll(w_group), _ll(o_group),
        _lib.ptr(order), _lib.ptr(start), _lib.ptr(count), a_div, groups, M, N, K, act, ctypes.c_float(cap),
        ctypes.c_float(second), N if act_cols is None else act_cols,
        int(A.dtype == torch.float32), int(out.dtype == torch.float32), typical, _lib.ptr(gate),
        _ll(0 if gate is None else gate.stride(0)), _ll(0 if gate is None else gate.stride(1)),
        0 if gate is None else gate.stride(2), row_tiles, _lib.stream_ptr())
    _lib.check(rc, "ts_skinny_gemm")


def _row_tiles(rows: int, cols: int) -> int:
    """Tiles of eight rows per pass when the passes run side by side: short passes while there are few of them (measured)."""
    return 1 if rows * cols <= 1 << 15 else 2


def rows_linear(x: torch.Tensor, w: torch.Tensor, out_dtype=None, act: int = ACT_NONE, cap: float = 0.0,
                out: torch.Tensor | None = None, second: float = 0.0, act_cols: int | None = None) -> torch.Tensor:
    """act(x [M, K] @ w [N, K]^T) for a handful of rows: the cost is one pass over w, spread over N / 16 CTAs."""
    if out is None:
        out = torch.empty(x.shape[0], w.shape[0] // (2 if is_gated(act) else 1), dtype=out_dtype or x.dtype, device=x.device)
    _launch(x, w, out, x.stride(0), w.stride(0), out.stride(0), 0, 0, 0, None, None, None, 1, 1, x.shape[0], w.shape[0],
            w.shape[1], act, cap=cap, row_tiles=_row_tiles(x.shape[0], w.shape[0]), second=second, act_cols=act_cols)
    return out


def head_linear(x: torch.Tensor, w: torch.Tensor, out: torch.Tensor | None = None, gate: torch.Tensor | None = None) -> torch.Tensor:
    """x [T, H, K] (last dimension contiguous), w [H, N, K] -> [T, H, N]: every head has its own matrix.  `gate` [T, H, N]
    (any strides, so it may be one number per head, expanded): the result is multiplied by sigmoid(gate)."""
    T, H, K = x.shape
    N = w.shape[1]
    if out is None:
        out = torch.empty(T, H, N, dtype=x.dtype, device=x.device)
    if not x.is_cuda:
        y = torch.einsum("thk,hnk->thn", x, w)
        return out.copy_(y if gate is None else y * torch.sigmoid(gate))
    _launch(x, w, out, x.stride(0), w.stride(1), out.stride(0), x.stride(1), w.stride(0), out.stride(1), None, None, None, 1,
            H, T, N, K, ACT_NONE, gate=gate, row_tiles=_row_tiles(T, H * N))
    return out


def expert_linear(x: torch.Tensor, w: torch.Tensor, order, start, count, slots: int, max_rows: int, per_row: int,
                  act: int = ACT_NONE) -> torch.Tensor:
    """out[s] = act(w[e(s)] @ x[s // per_row]) for every routed slot s; slots of expert e are
    order[start[e] : start[e] + count[e]].  w [E, N, K]; `max_rows` bounds count."""
    E, N, K = w.shape
    out = torch.empty(slots, N // (2 if is_gated(act) else 1), dtype=x.dtype, device=x.device)
    _launch(x, w, out, x.stride(0), w.stride(1), out.stride(0), 0, w.stride(0), 0, order, start, count, per_row, E, max_rows,
            N, K, act, -(-2 * slots // E), row_tiles=4)
    return out
