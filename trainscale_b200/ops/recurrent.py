"""Recurrent mixers with an fp32 matrix state per head: the gated delta rule (with short convolutions in front), WKV time
mixing (csrc/recurrent.cu) and retention (csrc/recurrent.cu; csrc/retention.cu for long portions).

All run over a flattened batch whose first rows are single tokens (decoding: one launch from projection to gated norm) and
whose other rows are portions of prompts (a scan).  A sequence's state row holds [convolution inputs or token-shift row, if any |
S of every head]; `rows.prev` / `rows.next` name the state rows a sequence continues from and leaves.  Tensors on the CPU
take PyTorch math.
"""
from __future__ import annotations

import ctypes
import functools
from dataclasses import dataclass

import torch
import torch.nn.functional as F

from . import _lib
from .stream import StreamRows

_ll, _f = ctypes.c_longlong, ctypes.c_float
MAX_HEAD = 256           # largest key or value size of a head
MAX_RETENTION_VALUE = 512  # retention: largest value size
RETENTION_CHUNK = 128      # tokens of a chunk of csrc/retention.cu
SCAN_WKV, SCAN_DELTA, SCAN_RETENTION = 0, 1, 2


def _up4(n: int) -> int:
    return -(-n // 4) * 4


@dataclass(frozen=True)
class DeltaShape:
    """Sizes of one gated delta rule mixer; its projection row is q | k | v | gate | beta | decay."""
    heads: int            # value heads
    kv_heads: int         # query / key heads
    dim: int
    vdim: int
    taps: int

    @property
    def channels(self) -> int:
        return 2 * self.kv_heads * self.dim + self.heads * self.vdim

    @property
    def proj_width(self) -> int:
        return self.channels + self.heads * self.vdim + 2 * self.heads

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def matrix_offset(self) -> int:
        return _up4((self.taps - 1) * self.channels)

    @property
    def state_width(self) -> int:
        return _up4(self.matrix_offset + self.heads * self.dim * self.vdim)


@dataclass(frozen=True)
class WkvShape:
    """Sizes of one WKV mixer; `width` is the model's (the token-shift row in front of the state)."""
    heads: int
    dim: int
    width: int

    @property
    def inner(self) -> int:
        return self.heads * self.dim

    @property
    def matrix_offset(self) -> int:
        return _up4(self.width)

    @property
    def state_width(self) -> int:
        return _up4(self.matrix_offset + self.heads * self.dim * self.dim)


@dataclass(frozen=True)
class RetentionShape:
    """Sizes and constants of one retention mixer; its projection row is q | k | v | gate."""
    heads: int
    dim: int
    vdim: int
    rot: int                       # rotated dimensions of a head
    decay: tuple[float, ...]       # per head

    @property
    def qk_width(self) -> int:
        return self.heads * self.dim

    @property
    def out_width(self) -> int:
        return self.heads * self.vdim

    @property
    def proj_width(self) -> int:
        return 2 * (self.qk_width + self.out_width)

    @property
    def state_width(self) -> int:
        return _up4(self.heads * self.dim * self.vdim)

    def powers(self) -> torch.Tensor:
        """fp32 [heads, RETENTION_CHUNK + 1] g^0, g^1, ... of the decays as fp32 numbers."""
        g = torch.tensor(self.decay, dtype=torch.float32).double()
        return (g[:, None] ** torch.arange(RETENTION_CHUNK + 1, dtype=torch.float64)).float()


@dataclass
class DeltaWeights:
    conv: torch.Tensor    # [channels, taps] fp32, last tap: the current token
    A_log: torch.Tensor   # [heads] fp32
    dt_bias: torch.Tensor
    norm: torch.Tensor    # [vdim] fp32, shared by heads


@dataclass
class WkvWeights:
    w0: torch.Tensor      # [heads * dim] fp32
    u: torch.Tensor       # [heads, dim] fp32
    norm: torch.Tensor    # [heads * dim] fp32


def _rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def _sequences(rows: StreamRows, n_single: int, cu: list[int], T: int):
    """(first row, end, state row read, state row written) of every single row and portion."""
    spans = [(i, i + 1) for i in range(n_single)] + [(n_single + a, n_single + b) for a, b in zip(cu[:-1], cu[1:])]
    for a, b in spans:
        yield a, b, int(rows.prev[a]), int(rows.next[b - 1])


# ---------------------------------------------------------------------------------------------- gated delta rule
def _delta_reference(proj, s: DeltaShape, w: DeltaWeights, eps, rows, state, n_single, cu, out, out_scale):
    C, kw = s.channels, s.kv_heads * s.dim
    rep = s.heads // s.kv_heads
    for a, b, prev, nxt in _sequences(rows, n_single, cu, proj.shape[0]):
        x = proj[a:b].float()
        tail = torch.zeros(s.taps - 1, C) if prev < 0 else state[prev, :(s.taps - 1) * C].view(s.taps - 1, C)
        S = torch.zeros(s.heads, s.dim, s.vdim) if prev < 0 else \
            state[prev, s.matrix_offset:s.matrix_offset + s.heads * s.dim * s.vdim].view(s.heads, s.dim, s.vdim)
        inp = torch.cat([tail, x[:, :C]])
        y = F.silu(sum(inp[j:j + b - a] * w.conv[:, j] for j in range(s.taps)))
        unit = lambda z: z / torch.sqrt(z.pow(2).sum(-1, keepdim=True) + 1e-6)   # noqa: E731
        q = (unit(y[:, :kw].view(-1, s.kv_heads, s.dim)) * s.dim ** -0.5).repeat_interleave(rep, 1)
        k = unit(y[:, kw:2 * kw].view(-1, s.kv_heads, s.dim)).repeat_interleave(rep, 1)
        v = y[:, 2 * kw:].view(-1, s.heads, s.vdim)
        at = C + s.out_width
        beta = torch.sigmoid(x[:, at:at + s.heads])
        g = torch.exp(-torch.exp(w.A_log) * F.softplus(x[:, at + s.heads:at + 2 * s.heads] + w.dt_bias))
        for t in range(b - a):
            S = g[t, :, None, None] * S
            u = beta[t, :, None] * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
            S = S + k[t, :, :, None] * u[:, None]
            o = _rms(torch.einsum("hdv,hd->hv", S, q[t]), eps) * w.norm
            out[a + t] = (o.reshape(-1) * F.silu(x[t, C:at]) * out_scale).to(out.dtype)
        if nxt >= 0:
            state[nxt, :(s.taps - 1) * C] = inp[b - a:].reshape(-1)
            state[nxt, s.matrix_offset:s.matrix_offset + S.numel()] = S.reshape(-1)


def delta_rule(proj: torch.Tensor, s: DeltaShape, w: DeltaWeights, eps: float, rows: StreamRows, state: torch.Tensor,
               n_single: int, portions, out: torch.Tensor, out_scale: float = 1.0) -> None:
    """proj [T, proj_width] (a column slice of a wider projection) -> out [T, heads * vdim] = out_scale * gated norm of the
    rule's result.  `portions`: offsets of the multi-token sequences after the `n_single` single rows (inference/batch)."""
    if not proj.is_cuda:
        return _delta_reference(proj, s, w, eps, rows, state, n_single, portions.offsets if portions else [0], out, out_scale)
    T = proj.shape[0]
    if n_single > 0:
        delta_step(proj[:n_single], s, w, eps, rows, state, out[:n_single], out_scale)
    if n_single < T:
        tail = StreamRows(rows.prev[n_single:], rows.next[n_single:])
        qkv, gates = delta_inputs(proj[n_single:], s, w, tail, state, portions)
        o = delta_scan(qkv, gates, s, tail, state, portions, proj.dtype == torch.bfloat16)
        gate = proj[n_single:, s.channels:s.channels + s.out_width]
        gated_norm(o, w.norm, 0, gate, out[n_single:], s.heads, s.vdim, eps, out_scale)


def delta_step(proj, s: DeltaShape, w: DeltaWeights, eps: float, rows: StreamRows, state, out, out_scale: float) -> None:
    """Single rows: convolution, norms, gates, state update, gated norm."""
    rc = _lib.load("recurrent").ts_delta_step(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(w.conv), _lib.ptr(w.A_log), _lib.ptr(w.dt_bias), _lib.ptr(w.norm),
        _f(eps), _f(s.dim ** -0.5), _lib.ptr(state), _ll(state.stride(0)), s.matrix_offset, _lib.ptr(rows.prev),
        _lib.ptr(rows.next), _lib.ptr(out), _ll(out.stride(0)), _f(out_scale), proj.shape[0], s.heads, s.kv_heads, s.dim,
        s.vdim, s.taps, int(proj.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_delta_step")


def delta_inputs(proj, s: DeltaShape, w: DeltaWeights, rows: StreamRows, state, portions):
    """Convolved and normed q | k | v [T, channels] and log decay | beta [T, 2 heads] of portions, both fp32."""
    T = proj.shape[0]
    qkv = torch.empty(T, s.channels, dtype=torch.float32, device=proj.device)
    gates = torch.empty(T, 2 * s.heads, dtype=torch.float32, device=proj.device)
    rc = _lib.load("recurrent").ts_delta_inputs(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(w.conv), _lib.ptr(w.A_log), _lib.ptr(w.dt_bias), _f(s.dim ** -0.5),
        _lib.ptr(state), _ll(state.stride(0)), _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(portions.cu),
        portions.count, portions.longest, _lib.ptr(qkv), _lib.ptr(gates), s.heads, s.kv_heads, s.dim, s.vdim, s.taps,
        int(proj.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_delta_inputs")
    return qkv, gates


@functools.lru_cache(maxsize=None)
def _blocked(dim: int, vdim: int) -> bool:
    return bool(_lib.load("recurrent").ts_block_scan_supported(dim, vdim))


def _workspace(T: int, portions, kind: int, *shape, device) -> torch.Tensor:
    """Uninitialised fp32 [blocks, heads, ...] for the per-block quantities of a block scan."""
    lib = _lib.load("recurrent")
    last = shape[1:] or (lib.ts_block_scan_coef(kind),)
    return torch.empty(lib.ts_block_scan_blocks(T, portions.count), shape[0], *last, dtype=torch.float32, device=device)


def delta_scan(qkv, gates, s: DeltaShape, rows: StreamRows, state, portions, blocked: bool = False) -> torch.Tensor:
    """The recurrence over portions: results [T, heads * vdim] fp32; leaves every portion's last state.  `blocked`: blocks of
    tokens on the tensor cores with split operands (head sizes that are multiples of 8), else plain fp32 arithmetic."""
    T = qkv.shape[0]
    o = torch.empty(T, s.out_width, dtype=torch.float32, device=qkv.device)
    if blocked and _blocked(s.dim, s.vdim):
        coef = _workspace(T, portions, SCAN_DELTA, s.heads, device=qkv.device)
        rc = _lib.load("recurrent").ts_delta_block_scan(
            _lib.ptr(qkv), _lib.ptr(gates), _lib.ptr(coef), _lib.ptr(state),
            _ll(state.stride(0)), s.matrix_offset, _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(portions.cu),
            portions.count, portions.longest, _lib.ptr(o), s.heads, s.kv_heads, s.dim, s.vdim, _lib.stream_ptr())
        _lib.check(rc, "ts_delta_block_scan")
        return o
    rc = _lib.load("recurrent").ts_delta_scan(
        _lib.ptr(qkv), _lib.ptr(gates), _lib.ptr(state), _ll(state.stride(0)), s.matrix_offset, _lib.ptr(rows.prev),
        _lib.ptr(rows.next), _lib.ptr(portions.cu), portions.count, _lib.ptr(o), s.heads, s.kv_heads, s.dim, s.vdim,
        _lib.stream_ptr())
    _lib.check(rc, "ts_delta_scan")
    return o


def gated_norm(o, w, w_head: int, gate, out, heads: int, vdim: int, eps: float, scale: float = 1.0) -> None:
    """out = o / rms per head * w * silu(gate) * scale; `w_head`: stride of w from head to head (0: shared); w None: one."""
    rc = _lib.load("recurrent").ts_gated_norm(
        _lib.ptr(o), _lib.ptr(w), w_head, _lib.ptr(gate), _ll(gate.stride(0)), _lib.ptr(out), _ll(out.stride(0)), o.shape[0],
        heads, vdim, _f(eps), _f(scale), int(out.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_gated_norm")


# ---------------------------------------------------------------------------------------------- WKV time mixing
def _wkv_reference(rkvg, w_raw, s: WkvShape, w: WkvWeights, eps, rows, state, n_single, cu, out):
    H, D = s.heads, s.dim
    for a, b, prev, nxt in _sequences(rows, n_single, cu, rkvg.shape[0]):
        at = s.matrix_offset
        S = torch.zeros(H, D, D) if prev < 0 else state[prev, at:at + H * D * D].view(H, D, D)
        r, k, v, gate = rkvg[a:b].float().unbind(1)
        r, k, v = (z.reshape(-1, H, D) for z in (r, k, v))
        decay = torch.exp(-torch.exp(w_raw[a:b] + w.w0)).view(-1, H, D)
        for t in range(b - a):
            kv = k[t, :, :, None] * v[t, :, None]
            o = torch.einsum("hdv,hd->hv", S + w.u[:, :, None] * kv, r[t])
            S = decay[t, :, :, None] * S + kv
            out[a + t] = (_rms(o, eps).reshape(-1) * w.norm * F.silu(gate[t])).to(out.dtype)
        if nxt >= 0:
            state[nxt, at:at + S.numel()] = S.reshape(-1)


def wkv(rkvg: torch.Tensor, w_raw: torch.Tensor, s: WkvShape, w: WkvWeights, eps: float, rows: StreamRows, state: torch.Tensor,
        n_single: int, portions, out: torch.Tensor) -> None:
    """rkvg [T, 4, inner] (r, k, v and the gate before its silu), w_raw [T, inner] fp32 (decay = exp(-exp(w_raw + w0))) ->
    out [T, inner], the gated norm of the recurrence."""
    if not rkvg.is_cuda:
        return _wkv_reference(rkvg, w_raw, s, w, eps, rows, state, n_single, portions.offsets if portions else [0], out)
    T = rkvg.shape[0]
    if n_single > 0:
        wkv_step(rkvg[:n_single], w_raw[:n_single], s, w, eps, rows, state, out[:n_single])
    if n_single < T:
        tail = StreamRows(rows.prev[n_single:], rows.next[n_single:])
        o = wkv_scan(rkvg[n_single:], w_raw[n_single:], s, w, tail, state, portions, rkvg.dtype == torch.bfloat16)
        gated_norm(o, w.norm, s.dim, rkvg[n_single:, 3], out[n_single:], s.heads, s.dim, eps)


def wkv_step(rkvg, w_raw, s: WkvShape, w: WkvWeights, eps: float, rows: StreamRows, state, out) -> None:
    rc = _lib.load("recurrent").ts_wkv_step(
        _lib.ptr(rkvg), _ll(rkvg.stride(0)), _lib.ptr(w_raw), _lib.ptr(w.w0), _lib.ptr(w.u), _lib.ptr(w.norm), _f(eps),
        _lib.ptr(state), _ll(state.stride(0)), s.matrix_offset, _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(out),
        _ll(out.stride(0)), rkvg.shape[0], s.heads, s.dim, int(rkvg.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_wkv_step")


def wkv_scan(rkvg, w_raw, s: WkvShape, w: WkvWeights, rows: StreamRows, state, portions, blocked: bool = False) -> torch.Tensor:
    """As `delta_scan`; `blocked` takes bf16 projections."""
    T, dev = rkvg.shape[0], rkvg.device
    o = torch.empty(T, s.inner, dtype=torch.float32, device=dev)
    if blocked and _blocked(s.dim, s.dim):
        rt, kt = (torch.empty(T, s.inner, dtype=torch.float32, device=dev) for _ in range(2))
        coef = _workspace(T, portions, SCAN_WKV, s.heads, device=dev)
        decay = _workspace(T, portions, SCAN_WKV, s.heads, s.dim, device=dev)
        rc = _lib.load("recurrent").ts_wkv_block_scan(
            _lib.ptr(rkvg), _ll(rkvg.stride(0)), _lib.ptr(w_raw), _lib.ptr(w.w0), _lib.ptr(w.u), _lib.ptr(rt), _lib.ptr(kt),
            _lib.ptr(coef), _lib.ptr(decay), _lib.ptr(state), _ll(state.stride(0)), s.matrix_offset, _lib.ptr(rows.prev),
            _lib.ptr(rows.next), _lib.ptr(portions.cu), portions.count, portions.longest, _lib.ptr(o), s.heads, s.dim,
            _lib.stream_ptr())
        _lib.check(rc, "ts_wkv_block_scan")
        return o
    rc = _lib.load("recurrent").ts_wkv_scan(
        _lib.ptr(rkvg), _ll(rkvg.stride(0)), _lib.ptr(w_raw), _lib.ptr(w.w0), _lib.ptr(w.u), _lib.ptr(state),
        _ll(state.stride(0)), s.matrix_offset, _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(portions.cu),
        portions.count, _lib.ptr(o), s.heads, s.dim, int(rkvg.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_wkv_scan")
    return o


# ---------------------------------------------------------------------------------------------- retention
def _turn(x: torch.Tensor, cs: torch.Tensor, rot: int) -> torch.Tensor:
    """x [T, H, D]: coordinate i turns with i + rot / 2; cs [T, rot] = cos | sin."""
    half = rot // 2
    c, s = cs[:, None, :half], cs[:, None, half:]
    u, v = x[..., :half], x[..., half:rot]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., rot:]], dim=-1)


def _retention_reference(proj, s: RetentionShape, powers, eps, cs, rows, state, n_single, cu, out):
    H, D, V, kw = s.heads, s.dim, s.vdim, s.qk_width
    g = powers[:, 1, None, None]
    for a, b, prev, nxt in _sequences(rows, n_single, cu, proj.shape[0]):
        x = proj[a:b].float()
        q, k = (_turn(z.reshape(b - a, H, D), cs[a:b], s.rot) for z in (x[:, :kw], x[:, kw:2 * kw]))
        k = k * D ** -0.5
        v, gate = x[:, 2 * kw:2 * kw + s.out_width].reshape(b - a, H, V), x[:, 2 * kw + s.out_width:s.proj_width]
        S = torch.zeros(H, D, V) if prev < 0 else state[prev, :H * D * V].view(H, D, V)
        for t in range(b - a):
            S = g * S + k[t, :, :, None] * v[t, :, None]
            o = _rms(torch.einsum("hdv,hd->hv", S, q[t]), eps)
            out[a + t] = (o.reshape(-1) * F.silu(gate[t])).to(out.dtype)
        if nxt >= 0:
            state[nxt, :S.numel()] = S.reshape(-1)


def retention(proj: torch.Tensor, s: RetentionShape, powers: torch.Tensor, eps: float, cs: torch.Tensor, rows: StreamRows,
              state: torch.Tensor, n_single: int, portions, out: torch.Tensor) -> None:
    """proj [T, >= proj_width] -> out [T, heads * vdim]: S <- g S + k v^T, o = S^T q with q and k rotated and k times dim^-1/2;
    o / rms per head * silu(gate).  cs fp32 [T, rot] of ops/window_attention.angles, powers of `RetentionShape.powers`."""
    if not proj.is_cuda:
        return _retention_reference(proj, s, powers, eps, cs, rows, state, n_single, portions.offsets if portions else [0], out)
    T = proj.shape[0]
    if n_single > 0:
        retention_step(proj[:n_single], s, powers, eps, cs, rows, state, out[:n_single])
    if n_single < T:
        tail = StreamRows(rows.prev[n_single:], rows.next[n_single:])
        part, bf16 = proj[n_single:], proj.dtype == torch.bfloat16
        if bf16 and portions.longest >= CHUNKS_FROM and _chunked(s.dim, s.vdim) and part.stride(0) % 8 == 0:
            return retention_chunks(part, s, powers, eps, cs[n_single:], tail, state, portions, out[n_single:])
        o = retention_scan(part, s, powers, cs[n_single:], tail, state, portions, bf16)
        gate = part[:, 2 * s.qk_width + s.out_width:s.proj_width]
        gated_norm(o, None, 0, gate, out[n_single:], s.heads, s.vdim, eps)


CHUNKS_FROM = 64         # tokens of the longest portion from which chunks side by side beat one block after another


@functools.lru_cache(maxsize=None)
def _chunked(dim: int, vdim: int) -> bool:
    return bool(_lib.load("retention").ts_retention_chunks_supported(dim, vdim))


def retention_chunks(proj, s: RetentionShape, powers, eps: float, cs, rows: StreamRows, state, portions, out) -> None:
    """Portions, bf16: from projection to gated norm, all chunks of a portion side by side."""
    lib, T = _lib.load("retention"), proj.shape[0]
    chunks = torch.empty(lib.ts_retention_chunks_count(T, portions.count), s.heads, s.dim, s.vdim, dtype=torch.float32, device=proj.device)
    rc = lib.ts_retention_chunks(
        _lib.ptr(proj), _ll(proj.stride(0)), _ll(T), _lib.ptr(cs), _lib.ptr(powers), powers.shape[1], _f(s.dim ** -0.5), _f(eps),
        _lib.ptr(chunks), _lib.ptr(state), _ll(state.stride(0)), _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(portions.cu),
        portions.count, portions.longest, _lib.ptr(out), _ll(out.stride(0)), s.heads, s.dim, s.vdim, s.rot, _lib.stream_ptr())
    _lib.check(rc, "ts_retention_chunks")


def retention_step(proj, s: RetentionShape, powers, eps: float, cs, rows: StreamRows, state, out) -> None:
    """Single rows: rotation, state update, norm and gate."""
    rc = _lib.load("recurrent").ts_retention_step(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(cs), _lib.ptr(powers), powers.shape[1], _f(s.dim ** -0.5), _f(eps), _lib.ptr(state),
        _ll(state.stride(0)), _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(out), _ll(out.stride(0)), proj.shape[0], s.heads,
        s.dim, s.vdim, s.rot, int(proj.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_retention_step")


def retention_scan(proj, s: RetentionShape, powers, cs, rows: StreamRows, state, portions, blocked: bool = False) -> torch.Tensor:
    """As `delta_scan`; `blocked` takes bf16 projections."""
    T, dev = proj.shape[0], proj.device
    o = torch.empty(T, s.out_width, dtype=torch.float32, device=dev)
    lib = _lib.load("recurrent")
    if blocked and _blocked(s.dim, s.vdim) and proj.stride(0) % 8 == 0:
        rt, kt = (torch.empty(T, s.qk_width, dtype=torch.float32, device=dev) for _ in range(2))
        coef = _workspace(T, portions, SCAN_RETENTION, s.heads, device=dev)
        rc = lib.ts_retention_block_scan(
            _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(cs), _lib.ptr(powers), powers.shape[1], _f(s.dim ** -0.5), _lib.ptr(rt), _lib.ptr(kt),
            _lib.ptr(coef), _lib.ptr(state), _ll(state.stride(0)), _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(portions.cu),
            portions.count, portions.longest, _lib.ptr(o), s.heads, s.dim, s.vdim, s.rot, _lib.stream_ptr())
        _lib.check(rc, "ts_retention_block_scan")
        return o
    rc = lib.ts_retention_scan(
        _lib.ptr(proj), _ll(proj.stride(0)), _lib.ptr(cs), _lib.ptr(powers), powers.shape[1], _f(s.dim ** -0.5), _lib.ptr(state),
        _ll(state.stride(0)), _lib.ptr(rows.prev), _lib.ptr(rows.next), _lib.ptr(portions.cu), portions.count, _lib.ptr(o), s.heads,
        s.dim, s.vdim, s.rot, int(proj.dtype == torch.float32), _lib.stream_ptr())
    _lib.check(rc, "ts_retention_scan")
    return o
