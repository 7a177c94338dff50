"""Kabulix: a pre-norm decoder whose layers mix with one of three kinds of attention and feed forward through a dense gated
product or a mixture of experts with a shared one; tied embedding.

    x <- x + mixer(n1(x)),  x <- x + ff(n2(x)),   n(x) = x / rms(x) * (1 + w),   logits = E n(x)
    attention         values are the (biased) keys before their norm and rotation; per-head norms, rotary pairs; a sliding
                      window that keeps the sequence's first tokens
    latent_attention  keys and values expanded from a normed latent, one rotary key part for all heads (YaRN frequencies);
                      a sliding window; result * sigmoid(gate), one gate per element
    attention_2       no positions; a token sees its chunk; result * sigmoid(gate), one gate per head
    dense             W_down (gelu(W_gate h) * W_up h)
    moe               sigmoid router over groups of experts, experts W_down (silu(W_gate h) * W_up h), and a shared expert of
                      the same form times sigmoid(W_sg h)
The sum of a sublayer's results (expert combine and shared factor included), the norm and the cast for the next GEMM are one
launch (ops/stream.prenorm); the stream is fp32.  Gates, biases and values ride in one input projection per mixer, the
shared factor in the router's.

A token leaves one row per layer in the paged cache - keys and values, or the latent and the rotated key part - and a
sequence has no other state, so prompts can share prefixes.  `serve` runs one flattened batch of decoding rows and portions
of prompts for the engine; sizes and constants come from the configuration and may differ per layer.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any

import torch
import torch.nn as nn

from ..ops import gemm, grouped, latent_attention as latent, moe, rope, stream, window_attention as window
from ..ops.grouped import GluRows, glu_width
from ..ops.latent_attention import LatentShape
from ..ops.moe import Router
from ..ops.window_attention import WindowShape
from .served import ServedDecoder, fp32_param, require, up8, weight_param

MAX_EXPERTS, MAX_TOP = 1024, 32


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    scaling: tuple[float, float, float, float] | None = None      # YaRN: factor, original, fast, slow

    def inv_freq(self) -> torch.Tensor:
        if self.scaling is None:
            return rope.rope_inv_freq(self.dims, self.base)
        factor, original, fast, slow = self.scaling
        return rope.rope_inv_freq(self.dims, self.base, "yarn", factor=factor, original_max_pos=original, beta_fast=fast,
                                  beta_slow=slow, ramp_end=self.dims - 1)

    @property
    def magnitude(self) -> float:
        return 1.0 if self.scaling is None else rope.yarn_magnitude(self.scaling[0])

    @classmethod
    def from_dict(cls, r: dict[str, Any]) -> "Rotation":
        s = r.get("scaling")
        return cls(r["dims"], float(r["base"]),
                   None if not s else tuple(float(s[k]) for k in ("factor", "original", "fast", "slow")))

    def to_dict(self) -> dict[str, Any]:
        d: dict[str, Any] = {"base": self.base, "dims": self.dims}
        if self.scaling is not None:
            d["scaling"] = dict(zip(("factor", "original", "fast", "slow"), self.scaling))
        return d


@dataclass(frozen=True)
class SinkConfig:
    """Mixer 'attention'."""
    shape: WindowShape
    rot: Rotation


@dataclass(frozen=True)
class LatentConfig:
    """Mixer 'latent_attention'."""
    shape: LatentShape
    rot: Rotation


@dataclass(frozen=True)
class ChunkConfig:
    """Mixer 'attention_2'."""
    shape: WindowShape


@dataclass(frozen=True)
class DenseConfig:
    ff: int


@dataclass(frozen=True)
class MoeConfig:
    router: Router
    ff: int
    shared_ff: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: SinkConfig | LatentConfig | ChunkConfig
    mlp: DenseConfig | MoeConfig | None


def _read_mixer(i: int, kind: str, m: dict[str, Any]):
    if kind not in ("attention", "latent_attention", "attention_2"):
        raise ValueError(f"layer {i}: unknown mixer {kind!r}")
    mask, scale = m["mask"], float(m["scale"])
    require(mask["size"] > 0 and mask.get("keep_first", 0) >= 0, i, "a window or chunk of at least one token")
    if kind == "latent_attention":
        rot = Rotation.from_dict(m["rot"])
        require(rot.dims == m["rot_dim"] and rot.dims % 2 == 0, i, "a rotation of the whole (even) rotated part of a head")
        return LatentConfig(LatentShape(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], mask["size"], scale,
                                        rot.base, True, rot.magnitude), rot)
    require(m["heads"] % m["kv_heads"] == 0, i, "whole head groups")
    if kind == "attention_2":
        return ChunkConfig(WindowShape(m["heads"], m["kv_heads"], m["dim"], m["vdim"], 0, mask["size"], scale, chunked=True))
    rot = Rotation.from_dict(m["rot"])
    require(rot.dims % 2 == 0 and rot.dims <= m["dim"], i, "an even number of rotated dimensions inside a head")
    require(m["vdim"] == m["dim"], i, "values of the size of the keys, which they are")
    return SinkConfig(WindowShape(m["heads"], m["kv_heads"], m["dim"], m["vdim"], rot.dims, mask["size"], scale,
                                  mask.get("keep_first", 0), pairs=True, values_are_keys=True), rot)


def _read_mlp(i: int, f: dict[str, Any] | None):
    if f is None:
        return None
    if f["kind"] == "dense":
        return DenseConfig(f["ff"])
    if f["kind"] != "moe":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    r = f["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    require(r["experts"] % g["count"] == 0 and 0 < g["keep"] <= g["count"], i, "equal groups of experts, some of them kept")
    require(0 < r["top"] <= g["keep"] * (r["experts"] // g["count"]), i, "no more experts per token than the kept groups hold")
    require(r["top"] <= MAX_TOP and r["experts"] <= MAX_EXPERTS, i, f"at most {MAX_TOP} of {MAX_EXPERTS} experts")
    return MoeConfig(Router(r["experts"], r["top"], True, g["count"], g["keep"]), f["expert"]["ff"], f["shared"]["ff"])


@dataclass(frozen=True)
class KabulixConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    layers: tuple[LayerConfig, ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "KabulixConfig":
        """Reads a config.json of this architecture."""
        layers = tuple(LayerConfig(_read_mixer(i, l["type"], l["mixer"]), _read_mlp(i, l.get("mlp")))
                       for i, l in enumerate(d["layers"]))
        if not layers:
            raise ValueError("a model needs layers")
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), layers)

    def to_dict(self) -> dict[str, Any]:
        layers = []
        for l in self.layers:
            s = l.mixer.shape
            mixer: dict[str, Any] = {"heads": s.heads, "dim": s.dim, "vdim": s.vdim, "scale": s.scale, "mask": {"size": s.window}}
            if isinstance(l.mixer, LatentConfig):
                kind = "latent_attention"
                mixer |= {"rot_dim": s.rot, "kv_rank": s.rank, "rot": l.mixer.rot.to_dict()}
            elif isinstance(l.mixer, SinkConfig):
                kind = "attention"
                mixer |= {"kv_heads": s.kv_heads, "rot": l.mixer.rot.to_dict()}
                mixer["mask"]["keep_first"] = s.keep
            else:
                kind = "attention_2"
                mixer["kv_heads"] = s.kv_heads
            mlp: dict[str, Any] | None = None
            if isinstance(l.mlp, DenseConfig):
                mlp = {"kind": "dense", "ff": l.mlp.ff}
            elif l.mlp is not None:
                r = l.mlp.router
                mlp = {"kind": "moe", "expert": {"ff": l.mlp.ff}, "shared": {"ff": l.mlp.shared_ff},
                       "router": {"experts": r.experts, "top": r.top, "groups": {"count": r.groups, "keep": r.keep}}}
            layers.append({"type": kind, "mixer": mixer, "mlp": mlp})
        return {"architecture": "Kabulix", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps},
                "layers": layers}


def pattern_config(kinds: str, vocab: int, width: int, heads: int, kv_heads: int, dim: int, window: int, keep: int, chunk: int,
                   latent_dim: int, latent_rot: int, latent_vdim: int, rank: int, latent_window: int, ff: int, experts: int, top: int,
                   expert_ff: int, shared_ff: int, groups: int, keep_groups: int, rot_dims: int | None = None,
                   rope_base: float = 10000.0, scaling: tuple[float, float, float, float] = (4.0, 4096.0, 32.0, 1.0),
                   dense_layers: int = 1, eps: float = 1e-6) -> KabulixConfig:
    """One layer per letter of `kinds`: w(indow with sinks), l(atent), c(hunks); the first `dense_layers` feed forward densely."""
    rot, yarn = Rotation(rot_dims or dim, rope_base), Rotation(latent_rot, rope_base, scaling)
    mixers = {
        "w": SinkConfig(WindowShape(heads, kv_heads, dim, dim, rot.dims, window, dim ** -0.5, keep, pairs=True, values_are_keys=True), rot),
        "l": LatentConfig(LatentShape(heads, latent_dim, latent_rot, latent_vdim, rank, latent_window, (latent_dim + latent_rot) ** -0.5,
                                      rope_base, True, yarn.magnitude), yarn),
        "c": ChunkConfig(WindowShape(heads, kv_heads, dim, dim, 0, chunk, dim ** -0.5, chunked=True))}
    sparse = MoeConfig(Router(experts, top, True, groups, keep_groups), expert_ff, shared_ff)
    return KabulixConfig(vocab, width, eps, tuple(LayerConfig(mixers[k], DenseConfig(ff) if i < dense_layers else sparse)
                                                  for i, k in enumerate(kinds)))


PRESETS: dict[str, KabulixConfig] = {
    "kabulix-tiny": pattern_config("wclw", vocab=32000, width=320, heads=4, kv_heads=2, dim=64, window=128, keep=4, chunk=192,
                                   latent_dim=64, latent_rot=32, latent_vdim=64, rank=96, latent_window=96, ff=640, experts=8, top=2,
                                   expert_ff=160, shared_ff=160, groups=4, keep_groups=2, rot_dims=32),
    "kabulix-3b": pattern_config("wclw" * 4, vocab=64000, width=2048, heads=16, kv_heads=4, dim=128, window=1024, keep=4, chunk=2048,
                                 latent_dim=128, latent_rot=64, latent_vdim=128, rank=512, latent_window=1024, ff=5504, experts=32,
                                 top=4, expert_ff=1024, shared_ff=1024, groups=8, keep_groups=4, rot_dims=64, rope_base=500000.0),
}


@dataclass
class StepContext:
    """What the layers of one step share."""
    positions: torch.Tensor
    row_len: torch.Tensor                       # keys of a row before the mask is applied
    side: "torch.cuda.Stream | None"            # captured decode: stream of the shared expert
    _angles: dict[Rotation, torch.Tensor] = field(default_factory=dict)

    def angles(self, rot: Rotation, inv_freq: torch.Tensor) -> torch.Tensor:
        if rot not in self._angles:
            self._angles[rot] = window.angles(inv_freq, self.positions, rot.magnitude)
        return self._angles[rot]


# ---------------------------------------------------------------------------------------------- mixers
class GroupedMixer(nn.Module):
    """Mixers 'attention' and 'attention_2'; projection row: q | k | v (unless the values are the keys) | gate per head."""

    def __init__(self, cfg: SinkConfig | ChunkConfig, width: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        s = cfg.shape
        self.sinks = isinstance(cfg, SinkConfig)
        self.w_in = weight_param(up8(s.in_width + (0 if self.sinks else s.heads)), width)
        self.w_o = weight_param(width, up8(s.out_width))
        self.bias = self.q_norm = self.k_norm = None
        if self.sinks:
            self.bias = fp32_param(s.q_width + s.kv_heads * s.dim)
            self.q_norm, self.k_norm = fp32_param(s.dim), fp32_param(s.dim)
            self.register_buffer("inv_freq", cfg.rot.inv_freq().to(self.q_norm.device), persistent=False)
        # columns of a projected row: what the GEMM writes, and room for the values where they come from the keys
        self.columns = max(self.w_in.shape[0], up8(s.q_width + s.kv_width))

    def tensors(self):
        """(checkpoint name under '.mix.', parameter or view of one)."""
        s = self.cfg.shape
        qw, kw, vw = s.q_width, s.kv_heads * s.dim, s.kv_heads * s.vdim
        yield "q", self.w_in[:qw]
        yield "k", self.w_in[qw:qw + kw]
        if self.sinks:
            yield "q.b", self.bias[:qw]
            yield "k.b", self.bias[qw:]
            yield "q.norm", self.q_norm
            yield "k.norm", self.k_norm
        else:
            yield "v", self.w_in[qw + kw:qw + kw + vw]
            yield "g", self.w_in[qw + kw + vw:qw + kw + vw + s.heads]
        yield "o", self.w_o[:, :s.out_width]

    def finalize(self) -> None:
        pass

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {"kv": (self.cfg.shape.row_width,)}

    def forward(self, h: torch.Tensor, batch, cache, ctx: StepContext) -> torch.Tensor:
        s, T, rows_cache = self.cfg.shape, h.shape[0], cache["kv"]
        proj = torch.empty(T, self.columns, dtype=h.dtype, device=h.device)
        gemm.serve_linear(h, self.w_in, out=proj[:, :self.w_in.shape[0]])
        gate = None if self.sinks else proj[:, s.in_width:s.in_width + s.heads]
        cs = ctx.angles(self.cfg.rot, self.inv_freq) if self.sinks else None
        window.prepare(proj, s, self.q_norm, self.k_norm, self.eps, cs, batch.slots, rows_cache, self.bias)
        out = torch.empty(T, self.w_o.shape[1], dtype=h.dtype, device=h.device)
        if s.out_width < out.shape[1]:
            out[:, s.out_width:] = 0
        tensor_cores = h.is_cuda and h.dtype == torch.bfloat16 and window.portions_supported(s)
        nd = batch.n_single if tensor_cores else T
        if nd > 0:
            window.attend_rows(proj[:nd], s, rows_cache, batch.block_table, batch.row_seq[:nd], ctx.row_len[:nd], batch.max_len,
                               out[:nd, :s.out_width], gate=None if gate is None else gate[:nd])
        if nd < T:
            keys = batch.prompt_context(s.mask)
            rows = None if keys.slots is None else latent.gather_rows(rows_cache, keys.slots)
            window.attend_portions(proj[nd:], s, rows, keys.cu_q, keys.cu_k, keys.max_q, out[nd:],
                                   gate=None if gate is None else gate[nd:])
        return gemm.serve_linear(out, self.w_o)


class LatentMixer(nn.Module):
    """Mixer 'latent_attention'; projection row: q | latent | rotated key part | padding | gate per element."""

    def __init__(self, cfg: LatentConfig, width: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        m = cfg.shape
        self.gate_at = up8(m.q_width + m.rank + m.rot)
        self.w_in = weight_param(up8(self.gate_at + m.heads * m.vdim), width)
        self.kv_norm = fp32_param(m.rank)
        self.w_kv = weight_param(m.heads * (m.dim + m.vdim), m.rank)          # unrotated keys | values, head by head
        self.w_o = weight_param(width, up8(m.heads * m.vdim))
        self.register_buffer("w_uk_t", torch.empty(m.heads, m.rank, m.dim), persistent=False)
        self.register_buffer("inv_freq", cfg.rot.inv_freq().to(self.kv_norm.device), persistent=False)

    def tensors(self):
        m = self.cfg.shape
        down = m.q_width + m.rank + m.rot
        yield "q", self.w_in[:m.q_width]
        yield "dkv", self.w_in[m.q_width:down]
        yield "g", self.w_in[self.gate_at:self.gate_at + m.heads * m.vdim]
        yield "dkv.norm", self.kv_norm
        yield "uk", self.w_kv[:m.heads * m.dim]
        yield "uv", self.w_kv[m.heads * m.dim:]
        yield "o", self.w_o[:, :m.heads * m.vdim]

    def finalize(self) -> None:
        """Derived weights: the key expansion transposed per head, for queries carried into latent space."""
        m = self.cfg.shape
        self.w_uk_t.copy_(self.w_kv[:m.heads * m.dim].view(m.heads, m.dim, m.rank).transpose(1, 2))

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {"latent": (self.cfg.shape.row_width,)}

    def forward(self, h: torch.Tensor, batch, cache, ctx: StepContext) -> torch.Tensor:
        m, T, rows_cache = self.cfg.shape, h.shape[0], cache["latent"]
        width = m.heads * m.vdim
        expanded = h.is_cuda and h.dtype == torch.bfloat16 and latent.expanded_supported(m)
        nd = batch.n_single if expanded else T
        proj = gemm.serve_linear(h, self.w_in)
        gate = proj[:, self.gate_at:self.gate_at + width]
        flat = latent.prepare(proj, m, self.kv_norm, self.eps, self.inv_freq, batch.positions, batch.slots, rows_cache, nd < T)
        out = torch.empty(T, self.w_o.shape[1], dtype=h.dtype, device=h.device)
        if width < out.shape[1]:
            out[:, width:] = 0
        if nd > 0:
            q = proj[:nd, :m.q_width].view(nd, m.heads, m.dim + m.rot)[..., :m.dim]
            o = latent.attend_latent(grouped.head_linear(q, self.w_uk_t), proj[:nd], m, rows_cache, batch.block_table,
                                     batch.row_seq[:nd], ctx.row_len[:nd], batch.max_len)
            w_uv = self.w_kv[m.heads * m.dim:].view(m.heads, m.vdim, m.rank)
            grouped.head_linear(o, w_uv, out[:nd, :width].unflatten(1, (m.heads, m.vdim)),
                                gate[:nd].unflatten(1, (m.heads, m.vdim)))
        if nd < T:
            keys = batch.prompt_context(m.mask)
            rows = flat[nd:] if keys.slots is None else latent.gather_rows(rows_cache, keys.slots)
            kv = gemm.matmul_nt(rows[:, :m.rank], self.w_kv)
            latent.attend_expanded(proj[nd:], kv, rows, m, keys.cu_q, keys.cu_k, keys.max_q, out[nd:], gate[nd:])
        return gemm.serve_linear(out, self.w_o)


# ---------------------------------------------------------------------------------------------- feed-forwards
class GatedProduct(nn.Module):
    """down(act(gate h) * up h), gate and up packed into one weight (ops/grouped)."""

    def __init__(self, width: int, ff: int, act: int):
        super().__init__()
        self.ff, self.act = ff, act
        self.w_in, self.w_down = weight_param(2 * glu_width(ff), width), weight_param(width, glu_width(ff))

    def tensors(self):
        yield "gate", GluRows(self.w_in, self.ff, 0)
        yield "up", GluRows(self.w_in, self.ff, 1)
        yield "down", self.w_down[:, :self.ff]

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return gemm.serve_linear(gemm.serve_linear(h, self.w_in, act=self.act), self.w_down)


class DenseFeedForward(nn.Module):
    def __init__(self, cfg: DenseConfig, width: int):
        super().__init__()
        self.product = GatedProduct(width, cfg.ff, grouped.ACT_GELU_GLU)

    def tensors(self):
        yield from self.product.tensors()

    def forward(self, h: torch.Tensor, ctx: StepContext):
        """(y, logits of a factor of y, routed experts) as ops/stream.prenorm takes them."""
        return self.product(h), None, None


class ExpertFeedForward(nn.Module):
    """Router rows: one per expert | the shared expert's factor | padding."""

    def __init__(self, cfg: MoeConfig, width: int):
        super().__init__()
        self.cfg = cfg
        E, F = cfg.router.experts, glu_width(cfg.ff)
        self.w_router = weight_param(up8(E + 1), width)
        self.w_in, self.w_down = weight_param(E, 2 * F, width), weight_param(E, width, F)
        self.shared = GatedProduct(width, cfg.shared_ff, grouped.ACT_SILU_GLU)

    def tensors(self):
        E, ff = self.cfg.router.experts, self.cfg.ff
        yield "router", self.w_router[:E]
        for e in range(E):
            yield f"e{e}.gate", GluRows(self.w_in[e], ff, 0)
            yield f"e{e}.up", GluRows(self.w_in[e], ff, 1)
            yield f"e{e}.down", self.w_down[e, :, :ff]
        for name, t in self.shared.tensors():
            yield f"shared.{name}", t
        yield "shared.sg", self.w_router[E:E + 1]

    def forward(self, h: torch.Tensor, ctx: StepContext):
        if ctx.side is not None:    # a captured decode step is a chain of short kernels: shared and routed experts at once
            main = torch.cuda.current_stream()
            ctx.side.wait_stream(main)
            with torch.cuda.stream(ctx.side):
                y = self.shared(h)
            logits, experts = self._routed(h)
            main.wait_stream(ctx.side)
        else:
            logits, experts = self._routed(h)
            y = self.shared(h)
        return y, logits[:, self.cfg.router.experts], experts

    def _routed(self, h: torch.Tensor):
        logits = gemm.serve_linear(h, self.w_router, torch.float32)
        return logits, moe.routed_experts(h, logits, self.w_in, self.w_down, self.cfg.router, grouped.ACT_SILU_GLU)


# ---------------------------------------------------------------------------------------------- the decoder
class KabulixLayer(nn.Module):
    def __init__(self, cfg: KabulixConfig, index: int):
        super().__init__()
        W, l = cfg.hidden_size, cfg.layers[index]
        self.norm1 = fp32_param(W)
        self.mixer = (LatentMixer if isinstance(l.mixer, LatentConfig) else GroupedMixer)(l.mixer, W, cfg.eps)
        self.ff = None
        if l.mlp is not None:
            self.norm2 = fp32_param(W)
            self.ff = (DenseFeedForward if isinstance(l.mlp, DenseConfig) else ExpertFeedForward)(l.mlp, W)


class KabulixForCausalLM(ServedDecoder):
    LIBRARIES = ("stream", "window", "latent", "latent_prefill", "skinny", "moe", "gemm")

    def __init__(self, cfg: KabulixConfig):
        super().__init__()
        self.config = cfg
        self.embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.hidden_size), requires_grad=False)
        self.layers = nn.ModuleList(KabulixLayer(cfg, i) for i in range(cfg.num_hidden_layers))
        self.final_norm = fp32_param(cfg.hidden_size)

    # ---------------------------------------------------------------- weights
    def _checkpoint_tensors(self):
        """(checkpoint name, parameter, view or packed part of one) of every stored tensor."""
        yield "embed", self.embed
        for i, l in enumerate(self.layers):
            yield f"l{i}.norm1", l.norm1
            for name, t in l.mixer.tensors():
                yield f"l{i}.mix.{name}", t
            if l.ff is not None:
                yield f"l{i}.norm2", l.norm2
                for name, t in l.ff.tensors():
                    yield f"l{i}.mlp.{name}", t
        yield "final.norm", self.final_norm

    @torch.no_grad()
    def reset_parameters(self, seed: int = 0) -> None:
        """Random weights from the parameters' own device generator (same device type and seed: same model)."""
        gen = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, t in self._checkpoint_tensors():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("norm1", "norm2", "b") or name == "final.norm":
                t.zero_()
            elif leaf == "norm":
                t.fill_(1.0)
            elif isinstance(t, GluRows):
                t.copy_(torch.empty(t.shape, dtype=torch.float32, device=gen.device).normal_(0.0, 1.0 / math.sqrt(t.shape[-1]), generator=gen))
            else:
                t.normal_(0.0, 1.0 / math.sqrt(t.shape[-1]), generator=gen)
        self.finalize()

    def finalize(self) -> None:
        for l in self.layers:
            l.mixer.finalize()

    # ---------------------------------------------------------------- serving interface of the engine
    def cache_spec(self):
        from ..inference.kv_cache import CacheSpec
        return CacheSpec([l.mixer.cache_entry() for l in self.layers])

    @torch.no_grad()
    def serve(self, batch, cache, observe=None) -> torch.Tensor:
        """Final-norm hidden state of the batch's wanted rows.  `observe(n, x)`: called with the stream after layer n (not
        the last)."""
        cfg, L, dtype = self.config, len(self.layers), self.embed.dtype
        ctx = StepContext(batch.positions, batch.positions + 1, self._side_stream() if batch.captured else None)
        x, h = stream.prenorm_embed(batch.token_ids, self.embed, self.layers[0].norm1, cfg.eps)
        for i, layer in enumerate(self.layers):
            add = layer.mixer(h, batch, cache.entries[i], ctx), None, None
            if layer.ff is not None:
                x, h = stream.prenorm(x, *add, layer.norm2, cfg.eps, dtype)
                add = layer.ff(h, ctx)
            if i + 1 == L:
                break
            x, h = stream.prenorm(x, *add, self.layers[i + 1].norm1, cfg.eps, dtype)
            if observe is not None:
                observe(i, x)
        return stream.prenorm_final(x, *add, self.final_norm, cfg.eps, batch.out_rows, dtype)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return gemm.serve_linear(hidden, self.embed, torch.float32)


def build_model(config, dtype=torch.bfloat16, device=None, seed: int | None = None) -> KabulixForCausalLM:
    """Randomly initialised model of a preset name, a config.json dictionary or a KabulixConfig."""
    if isinstance(config, str):
        config = PRESETS[config]
    elif isinstance(config, dict):
        config = KabulixConfig.from_dict(config)
    return KabulixForCausalLM.random(config, dtype, device, seed)


def load_model(config: dict, state_dict: dict[str, torch.Tensor], dtype=torch.bfloat16, device=None) -> KabulixForCausalLM:
    return KabulixForCausalLM.from_checkpoint(KabulixConfig.from_dict(config), state_dict, dtype, device)
