"""Device-side mixture-of-experts dataflow: routing plan, permute, grouped expert GEMMs, weighted combine.

Tokens are sorted by expert into a buffer whose per-expert segments start on 128-row boundaries (pad rows are zero), so
one persistent tcgen05 GEMM launch serves all experts (`ts_gemm_grouped_bf16`): every 128-row tile reads the weight
slab of its expert.  Nothing here synchronises with the host: buffer sizes use the static upper bound
`ts_moe_padded_rows(n, E)`.

Reference: data_pipeline/trainer/kernels/moe_kernels.py:219-785 (grouped GEMM, permute, top-k weighting) with the
per-expert loop of :1183 as the oracle.
"""
from __future__ import annotations

import ctypes
from dataclasses import dataclass

import torch

from . import _lib, activation

_c = ctypes


@dataclass
class MoEPlan:
    n: int                    # routed slots (tokens * top_k)
    k: int
    E: int
    P: int                    # rows of the padded expert-sorted buffer (static upper bound)
    counts: torch.Tensor      # [E] int32
    seg_start: torch.Tensor   # [E + 1] int32, multiples of 128
    tile_expert: torch.Tensor  # [P / 128] int32, -1 for unused tiles
    dest: torch.Tensor        # [n] int32: row of slot i
    src_of_row: torch.Tensor  # [P] int32: slot of row r or -1


def available(x: torch.Tensor) -> bool:
    return x.is_cuda and x.dtype == torch.bfloat16 and x.shape[-1] % 8 == 0


def make_plan(expert_ids: torch.Tensor, num_experts: int) -> MoEPlan:
    """expert_ids [T, k] (any integer dtype) -> routing plan; stable order inside every expert."""
    lib = _lib.load("moe")
    T, k = expert_ids.shape
    ids = expert_ids.reshape(-1).to(torch.int32).contiguous()
    n, E = ids.numel(), int(num_experts)
    P = int(lib.ts_moe_padded_rows(n, E))
    dev = ids.device
    i32 = dict(dtype=torch.int32, device=dev)
    rank, counts, seg = torch.empty(n, **i32), torch.empty(E, **i32), torch.empty(E + 1, **i32)
    tile_expert, dest, src = torch.empty(P // 128, **i32), torch.empty(n, **i32), torch.empty(P, **i32)
    rc = lib.ts_moe_plan(_lib.ptr(ids), n, E, _lib.ptr(rank), _lib.ptr(counts), _lib.ptr(seg), _lib.ptr(tile_expert),
                         _lib.ptr(dest), _lib.ptr(src), _lib.stream_ptr())
    _lib.check(rc, "ts_moe_plan")
    return MoEPlan(n, k, E, P, counts, seg, tile_expert, dest, src)


def _permute_raw(x2, plan: MoEPlan, slot_scale=None):
    lib = _lib.load("moe")
    out = torch.empty(plan.P, x2.shape[1], dtype=x2.dtype, device=x2.device)
    rc = lib.ts_moe_permute(_lib.ptr(x2), _lib.ptr(plan.src_of_row), _lib.ptr(slot_scale), _lib.ptr(out), plan.P,
                            x2.shape[1], plan.k, _lib.stream_ptr())
    _lib.check(rc, "ts_moe_permute")
    return out


def _combine_raw(y, plan: MoEPlan, w=None):
    lib = _lib.load("moe")
    T = plan.n // plan.k
    out = torch.empty(T, y.shape[1], dtype=y.dtype, device=y.device)
    rc = lib.ts_moe_combine(_lib.ptr(y), _lib.ptr(plan.dest), _lib.ptr(w), _lib.ptr(out), T, y.shape[1], plan.k,
                            _lib.stream_ptr())
    _lib.check(rc, "ts_moe_combine")
    return out


class _PermuteFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, x2, plan):
        ctx.plan = plan
        return _permute_raw(x2.contiguous(), plan)

    @staticmethod
    def backward(ctx, dxp):
        return _combine_raw(dxp.contiguous(), ctx.plan), None


class _CombineFn(torch.autograd.Function):
    @staticmethod
    def forward(ctx, y, w, plan):
        wf = w.reshape(-1).float().contiguous()
        ctx.save_for_backward(y, wf)
        ctx.plan, ctx.w_dtype, ctx.w_shape = plan, w.dtype, w.shape
        return _combine_raw(y.contiguous(), plan, wf)

    @staticmethod
    def backward(ctx, dout):
        lib = _lib.load("moe")
        y, wf = ctx.saved_tensors
        plan = ctx.plan
        dout = dout.contiguous()
        dy = _permute_raw(dout, plan, wf)                         # dy[dest(t, j)] = w[t, j] * dout[t]; pad rows zero
        dw = torch.empty(plan.n, dtype=torch.float32, device=y.device)
        rc = lib.ts_moe_combine_dw(_lib.ptr(dout), _lib.ptr(y), _lib.ptr(plan.dest), _lib.ptr(dw), plan.n, y.shape[1],
                                   plan.k, _lib.stream_ptr())
        _lib.check(rc, "ts_moe_combine_dw")
        return dy, dw.view(ctx.w_shape).to(ctx.w_dtype), None


def _grouped(mode, A, B, out, M, N, K, lda, ldb, ldc, a_mn, b_mn, accumulate, groups, E):
    lib = _lib.load("gemm")
    rc = lib.ts_gemm_grouped_bf16(_lib.ptr(A), _lib.ptr(B), _lib.ptr(out), mode, M, N, K, lda, ldb, ldc, int(a_mn),
                                  int(b_mn), int(out.dtype == torch.float32), int(accumulate), _c.c_float(1.0),
                                  _lib.ptr(groups), E, _lib.stream_ptr())
    _lib.check(rc, "ts_gemm_grouped_bf16")
    _lib.LAUNCHES += 1


class _GroupedLinearFn(torch.autograd.Function):
    """y[r] = x[r] @ W[e(r)]^T on the padded expert-sorted buffer; W is [E, N, K]."""

    @staticmethod
    def forward(ctx, xp, W, plan):
        E, N, K = W.shape
        y = torch.empty(plan.P, N, dtype=xp.dtype, device=xp.device)
        _grouped(1, xp, W, y, plan.P, N, K, K, K, N, False, False, False, plan.tile_expert, E)
        # rows of unused tiles (tile_expert == -1) are never written nor read back by the combine
        ctx.save_for_backward(xp, W)
        ctx.plan = plan
        return y

    @staticmethod
    def backward(ctx, dy):
        xp, W = ctx.saved_tensors
        plan = ctx.plan
        E, N, K = W.shape
        dy = dy.contiguous()
        dx = dW = None
        if ctx.needs_input_grad[0]:
            dx = torch.empty_like(xp)
            # dx[r] = dy[r] @ W[e]: B = W stacked along the reduction axis ([E*N][K], N-contiguous rows are K wide)
            _grouped(1, dy, W, dx, plan.P, K, N, N, K, K, False, True, False, plan.tile_expert, E)
        if ctx.needs_input_grad[1]:
            main_grad = getattr(W, "main_grad", None)
            if main_grad is not None:
                tgt, acc = main_grad.view(W.shape), bool(getattr(W, "grad_added", False))
                W.grad_added = True
            else:
                tgt, acc = torch.empty_like(W), False
            # dW[e] = dy_seg^T @ x_seg, reduced over the expert's row segment
            _grouped(2, dy, xp, tgt, N, K, plan.P, N, K, K, True, True, acc, plan.seg_start, E)
            dW = None if main_grad is not None else tgt
        return dx, dW, None


def grouped_linear(xp: torch.Tensor, W: torch.Tensor, plan: MoEPlan) -> torch.Tensor:
    return _GroupedLinearFn.apply(xp, W, plan)


def moe_ffn(x2: torch.Tensor, expert_ids: torch.Tensor, weights: torch.Tensor, w_gate_up: torch.Tensor,
            w_down: torch.Tensor, act: str = "silu") -> torch.Tensor:
    """Top-k expert feed-forward: out[t] = sum_j weights[t, j] * FFN_{ids[t, j]}(x2[t]).
    w_gate_up [E, 2I, H], w_down [E, H, I]."""
    plan = make_plan(expert_ids, w_gate_up.shape[0])
    xp = _PermuteFn.apply(x2, plan)
    h = grouped_linear(xp, w_gate_up, plan)
    h = activation.glu(h, act)
    y = grouped_linear(h, w_down, plan)
    return _CombineFn.apply(y, weights, plan)


def moe_ffn_reference(x2: torch.Tensor, expert_ids: torch.Tensor, weights: torch.Tensor, w_gate_up: torch.Tensor,
                      w_down: torch.Tensor, act: str = "silu") -> torch.Tensor:
    """Same result as `moe_ffn` by a loop over the experts (fp32 accumulation); differentiable.  CPU / non-bf16 path."""
    out = torch.zeros(x2.shape, dtype=torch.float32, device=x2.device)
    for e in range(w_gate_up.shape[0]):
        tok, slot = (expert_ids == e).nonzero(as_tuple=True)
        if tok.numel():
            h = activation.glu(x2[tok].float() @ w_gate_up[e].float().t(), act)
            out = out.index_add(0, tok, (h @ w_down[e].float().t()) * weights[tok, slot].float().unsqueeze(1))
    return out.to(x2.dtype)


class _TopKSoftmaxFn(torch.autograd.Function):
    """Router softmax + top-k on the device kernel; the (small, [T, E]) backward is written with torch ops."""

    @staticmethod
    def forward(ctx, logits, k, normalize):
        lib = _lib.load("moe")
        T, E = logits.shape
        lg = logits.float().contiguous()
        probs = torch.empty_like(lg)
        w = torch.empty(T, k, dtype=torch.float32, device=lg.device)
        idx = torch.empty(T, k, dtype=torch.int32, device=lg.device)
        rc = lib.ts_moe_topk_softmax(_lib.ptr(lg), _lib.ptr(probs), _lib.ptr(w), _lib.ptr(idx), T, E, int(k),
                                     int(bool(normalize)), _lib.stream_ptr())
        _lib.check(rc, "ts_moe_topk_softmax")
        idx64 = idx.long()
        ctx.save_for_backward(probs, w, idx64)
        ctx.normalize, ctx.in_dtype = bool(normalize), logits.dtype
        ctx.mark_non_differentiable(idx64)
        return w, idx64, probs

    @staticmethod
    def backward(ctx, dw, _didx, dprobs):
        probs, w, idx = ctx.saved_tensors
        dp = torch.zeros_like(probs) if dprobs is None else dprobs.float().clone()
        if dw is not None:
            dw = dw.float()
            if ctx.normalize:
                raw = probs.gather(1, idx)
                s = raw.sum(-1, keepdim=True).clamp(min=1e-9)
                dsel = (dw - (dw * w).sum(-1, keepdim=True)) / s
            else:
                dsel = dw
            dp.scatter_add_(1, idx, dsel)
        dlogits = probs * (dp - (dp * probs).sum(-1, keepdim=True))
        return dlogits.to(ctx.in_dtype), None, None


def topk_softmax(logits: torch.Tensor, k: int, normalize: bool = True):
    """(weights [T, k] fp32, experts [T, k] int64, probs [T, E] fp32) of the router logits."""
    if logits.is_cuda and logits.shape[1] <= 1024 and k <= 32:
        return _TopKSoftmaxFn.apply(logits, k, normalize)
    probs = torch.softmax(logits.float(), dim=-1)
    w, idx = probs.topk(k, dim=-1)
    if normalize:
        w = w / w.sum(-1, keepdim=True).clamp(min=1e-9)
    return w, idx, probs


# ---------------------------------------------------------------------------------------------- serving (no autograd)
# up to this many tokens and routed slots the experts are read by the few-row kernels instead of 128-row tiles (measured)
DECODE_ROWS, DECODE_SLOTS = 64, 128


@dataclass(frozen=True)
class Router:
    """How logits become the chosen experts and their weights.  `groups` 0: softmax over all experts, the `top` largest.
    Else sigmoid scores; experts form `groups` equal groups of neighbours, and only those of the `keep` groups with the
    largest sums of their two largest scores can be chosen."""
    experts: int
    top: int
    normalize: bool = False
    groups: int = 0
    keep: int = 0

    def choose(self, logits: torch.Tensor) -> tuple[torch.Tensor, torch.Tensor]:
        """(weights [T, top] fp32, experts [T, top]) in PyTorch math."""
        z = logits[:, :self.experts].float()
        if self.groups == 0:
            return topk_softmax(z, self.top, self.normalize)[:2]
        s = torch.sigmoid(z)
        size = self.experts // self.groups
        value = s.unflatten(1, (self.groups, size)).topk(min(2, size), dim=-1).values.sum(-1)
        best = torch.zeros_like(value, dtype=torch.bool).scatter_(1, value.topk(self.keep, dim=-1).indices, True)
        w, idx = s.masked_fill(~best.repeat_interleave(size, dim=1), -1.0).topk(self.top, dim=-1)
        return (w / (w.sum(-1, keepdim=True) + 1e-20) if self.normalize else w), idx


def _topk_raw(logits: torch.Tensor, r: Router):
    T, k = logits.shape[0], r.top
    w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    idx = torch.empty(T, k, dtype=torch.int32, device=logits.device)
    rc = _lib.load("moe").ts_moe_topk(_lib.ptr(logits), _c.c_longlong(logits.stride(0)), _lib.ptr(None), _lib.ptr(w),
                                      _lib.ptr(idx), T, r.experts, k, int(r.normalize), r.groups, r.keep, _lib.stream_ptr())
    _lib.check(rc, "ts_moe_topk")
    return w, idx


def _route_decode(logits: torch.Tensor, r: Router):
    T, E, k = logits.shape[0], r.experts, r.top
    i32 = dict(dtype=torch.int32, device=logits.device)
    w = torch.empty(T, k, dtype=torch.float32, device=logits.device)
    order, start, count = torch.empty(T * k, **i32), torch.empty(E, **i32), torch.empty(E, **i32)
    rc = _lib.load("moe").ts_moe_route(_lib.ptr(logits), _c.c_longlong(logits.stride(0)), _lib.ptr(w), _lib.ptr(order),
                                       _lib.ptr(start), _lib.ptr(count), T, E, k, int(r.normalize), r.groups, r.keep,
                                       _lib.stream_ptr())
    _lib.check(rc, "ts_moe_route")
    return w, order, start, count


def _grouped_act(x, W, plan: MoEPlan, act: int):
    from .grouped import is_gated
    E, N, K = W.shape
    cols = N // 2 if is_gated(act) else N
    y = torch.empty(plan.P, cols, dtype=x.dtype, device=x.device)
    rc = _lib.load("gemm").ts_gemm_grouped_bf16_act(
        _lib.ptr(x), _lib.ptr(W), _lib.ptr(y), 1, plan.P, N, K, K, K, cols, 0, 0, 0, 0, _c.c_float(1.0),
        _lib.ptr(plan.tile_expert), E, act, _lib.stream_ptr())
    _lib.check(rc, "ts_gemm_grouped_bf16_act")
    return y


def routed_experts(x: torch.Tensor, logits: torch.Tensor, w_up: torch.Tensor, w_down: torch.Tensor, router: Router | int, act: int):
    """Experts down(act(up x)) that the router chooses for every token, NOT combined: the layer boundary sums them into the
    fp32 stream.  x [T, H], logits [T, >= E] fp32, w_up [E, F, H], w_down [E, H, F], act of ops/grouped (gated: w_up is
    packed, [E, 2 F, H]); a number k as router is the k largest of a softmax.
    Returns (outputs, dest, weights [T, k]): slot t * k + j is row dest[slot] of the outputs (dest None: row slot).

    Few tokens: router, top-k and sort in one kernel, then one pass over the visited experts' weights.  Many (bf16):
    128-row expert segments on the grouped tcgen05 GEMM, the activation in its epilogue."""
    from . import grouped
    if isinstance(router, int):
        router = Router(w_up.shape[0], router)
    T, E, k = x.shape[0], router.experts, router.top
    if not x.is_cuda:
        w, idx = router.choose(logits)
        y = torch.zeros(T * k, x.shape[1], dtype=x.dtype)
        for e in range(E):
            slots = (idx.reshape(-1) == e).nonzero().squeeze(1)
            y[slots] = grouped.activate(x[slots // k] @ w_up[e].t(), act) @ w_down[e].t()
        return y, None, w
    H, F = x.shape[1], w_down.shape[2]
    if T <= DECODE_ROWS and T * k <= DECODE_SLOTS:
        w, order, start, count = _route_decode(logits, router)
    else:
        w, idx = _topk_raw(logits, router)
        plan = make_plan(idx, E)
        if x.dtype == torch.bfloat16 and H % 8 == 0 and F % 8 == 0:
            h = _grouped_act(_permute_raw(x, plan), w_up, plan, act)
            return _grouped_act(h, w_down, plan, grouped.ACT_NONE), plan.dest, w
        order, start, count = plan.src_of_row, plan.seg_start, plan.counts
    h = grouped.expert_linear(x, w_up, order, start, count, T * k, T, k, act)
    return grouped.expert_linear(h, w_down, order, start, count, T * k, T, 1), None, w
