"""Lovurax: a pre-norm decoder whose layers mix with retention, with sigmoid attention or with latent attention; a gate per element
on every sublayer's result; dense xIELU feed-forwards; tied embedding and scaled logits.

    x <- x + mixer(n1(x)) * sigmoid(G1 n1(x) + b1),  x <- x + ff(n2(x)) * sigmoid(G2 n2(x) + b2),   n(x) = x / rms(x) * w
    logits = c E n(x)
    retention         S <- g S + k v^T,  o = S^T q, one constant decay per head; q and k rotated by halves; o / rms * silu(gate)
    attention         grouped queries, head norms, a query factor that grows with the position; no rotation: a head's slope times
                      the distance is taken off its scores; weights sigmoid(score + bias), not normalized; result * sigmoid(gate),
                      one gate per element
    latent_attention  keys and values expanded from a normed latent, no positions; softmax; result * sigmoid(gate), one per head
    dense             W_down xielu(W_up h)
The gated sum of a sublayer's result, the norm and the cast for the next GEMM are one launch (ops/stream.prenorm); the stream is
fp32.  A mixer's gates and its residual gate ride in its input projection, that of a feed-forward in the up projection, whose
activation stops before it.

A token leaves keys and values or a latent per attending layer in the paged cache; a sequence has one fp32 matrix per retention
head in its state rows.  `serve` runs one flattened batch of decoding rows and portions of prompts for the engine; sizes and
constants come from the configuration and may differ per layer.
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any

import torch
import torch.nn as nn

from ..ops import gemm, grouped, latent_attention as latent, recurrent, rope, stream, window_attention as window
from ..ops.latent_attention import LatentShape
from ..ops.masks import UNBOUNDED
from ..ops.recurrent import RetentionShape
from ..ops.stream import ElementGate
from ..ops.window_attention import ScoreBias, WindowShape
from .served import ServedDecoder, fp32_param, require, up8, weight_param

RANDOM_SCORE_ADD = -4.0        # of a randomly initialised attention mixer


@dataclass(frozen=True)
class RetentionConfig:
    """Mixer 'retention'."""
    shape: RetentionShape
    base: float               # of the rotation


@dataclass(frozen=True)
class AttentionConfig:
    """Mixer 'attention'."""
    shape: WindowShape


@dataclass(frozen=True)
class LatentConfig:
    """Mixer 'latent_attention'."""
    shape: LatentShape


@dataclass(frozen=True)
class LayerConfig:
    mixer: RetentionConfig | AttentionConfig | LatentConfig
    ff: int | None


def _read_mixer(i: int, kind: str, m: dict[str, Any]):
    if kind == "retention":
        rot, decay = m["rot"], tuple(float(d) for d in m["decay"])
        require(rot["dims"] % 2 == 0 and rot["dims"] <= m["dim"], i, "an even number of rotated dimensions inside a head")
        require(len(decay) == m["heads"], i, "a decay for every head")
        require(m["dim"] <= recurrent.MAX_HEAD and m["vdim"] <= recurrent.MAX_RETENTION_VALUE, i,
                f"heads of up to {recurrent.MAX_HEAD} key and {recurrent.MAX_RETENTION_VALUE} value dimensions")
        return RetentionConfig(RetentionShape(m["heads"], m["dim"], m["vdim"], rot["dims"], decay), float(rot["base"]))
    if kind == "attention":
        t = m["q_temp"]
        require(m["heads"] % m["kv_heads"] == 0, i, "whole head groups")
        require(int(t["every"]) == t["every"] and t["every"] > 0, i, "a query temperature that grows every so many whole tokens")
        return AttentionConfig(WindowShape(m["heads"], m["kv_heads"], m["dim"], m["vdim"], 0, UNBOUNDED, float(m["scale"]),
                                           sigmoid=True, temperature=(float(t["coef"]), int(t["every"]))))
    if kind == "latent_attention":
        return LatentConfig(LatentShape(m["heads"], m["dim"], 0, m["vdim"], m["kv_rank"], UNBOUNDED, float(m["scale"])))
    raise ValueError(f"layer {i}: unknown mixer {kind!r}")


def _read_mlp(i: int, f: dict[str, Any] | None) -> int | None:
    if f is not None and f["kind"] != "dense":
        raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
    return None if f is None else f["ff"]


@dataclass(frozen=True)
class LovuraxConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    logit_scale: float
    layers: tuple[LayerConfig, ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "LovuraxConfig":
        """Reads a config.json of this architecture."""
        layers = tuple(LayerConfig(_read_mixer(i, l["type"], l["mixer"]), _read_mlp(i, l.get("mlp")))
                       for i, l in enumerate(d["layers"]))
        if not layers:
            raise ValueError("a model needs layers")
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), float(d["logit_scale"]), layers)

    def to_dict(self) -> dict[str, Any]:
        layers = []
        for l in self.layers:
            s = l.mixer.shape
            mixer: dict[str, Any] = {"heads": s.heads, "dim": s.dim, "vdim": s.vdim}
            if isinstance(l.mixer, RetentionConfig):
                kind = "retention"
                mixer |= {"decay": list(s.decay), "rot": {"base": l.mixer.base, "dims": s.rot}}
            elif isinstance(l.mixer, AttentionConfig):
                kind = "attention"
                mixer |= {"kv_heads": s.kv_heads, "scale": s.scale, "q_temp": dict(zip(("coef", "every"), s.temperature))}
            else:
                kind = "latent_attention"
                mixer |= {"kv_rank": s.rank, "scale": s.scale}
            layers.append({"type": kind, "mixer": mixer, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": "Lovurax", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps},
                "logit_scale": self.logit_scale, "layers": layers}


def pattern_config(kinds: str, vocab: int, width: int, heads: int, kv_heads: int, dim: int, ret_heads: int, ret_dim: int,
                   ret_vdim: int, latent_dim: int, latent_vdim: int, rank: int, ff: int, rope_base: float = 10000.0,
                   temperature: tuple[float, int] = (0.1, 4096), eps: float = 1e-6, logit_scale: float = 1.0) -> LovuraxConfig:
    """One layer per letter of `kinds`: r(etention), a(ttention), l(atent).  Decays 1 - 2^-(5 + h), their exponents spread over
    5 .. 12 whatever the number of heads."""
    decay = tuple(1.0 - 2.0 ** -(5 + 7 * h / max(1, ret_heads - 1)) for h in range(ret_heads))
    mixers = {
        "r": RetentionConfig(RetentionShape(ret_heads, ret_dim, ret_vdim, ret_dim, decay), rope_base),
        "a": AttentionConfig(WindowShape(heads, kv_heads, dim, dim, 0, UNBOUNDED, dim ** -0.5, sigmoid=True, temperature=temperature)),
        "l": LatentConfig(LatentShape(heads, latent_dim, 0, latent_vdim, rank, UNBOUNDED, latent_dim ** -0.5))}
    return LovuraxConfig(vocab, width, eps, logit_scale, tuple(LayerConfig(mixers[k], ff) for k in kinds))


PRESETS: dict[str, LovuraxConfig] = {
    "lovurax-tiny": pattern_config("rarl", vocab=32000, width=256, heads=4, kv_heads=2, dim=64, ret_heads=2, ret_dim=64, ret_vdim=128,
                                   latent_dim=64, latent_vdim=64, rank=96, ff=640, temperature=(0.2, 64)),
    "lovurax-2b": pattern_config("rarl" * 5, vocab=64000, width=2048, heads=16, kv_heads=4, dim=128, ret_heads=8, ret_dim=128,
                                 ret_vdim=256, latent_dim=128, latent_vdim=128, rank=512, ff=8192, rope_base=500000.0),
}


@dataclass
class StepContext:
    """What the layers of one step share."""
    rows: stream.StreamRows
    positions: torch.Tensor
    row_len: torch.Tensor                       # keys of a row
    _angles: dict[tuple[int, float], torch.Tensor] = field(default_factory=dict)

    def angles(self, rot: tuple[int, float], inv_freq: torch.Tensor) -> torch.Tensor:
        if rot not in self._angles:
            self._angles[rot] = window.angles(inv_freq, self.positions)
        return self._angles[rot]


# ---------------------------------------------------------------------------------------------- mixers
class Mixer(nn.Module):
    """Projection row: what the mixer reads (`in_width` columns) | padding | its residual gate | padding."""

    def __init__(self, in_width: int, out_width: int, width: int, eps: float):
        super().__init__()
        self.eps, self.width, self.out_width, self.gate_at = eps, width, out_width, up8(in_width)
        self.w_in = weight_param(up8(self.gate_at + width), width)
        self.w_o = weight_param(width, up8(out_width))
        self.gate_bias = fp32_param(width)

    def _rows(self, **sizes: int):
        """(name, rows of the input projection) one after the other."""
        at = 0
        for name, n in sizes.items():
            yield name, self.w_in[at:at + n]
            at += n

    def residual_gate(self):
        """(checkpoint name behind 'rg1', parameter) of the residual gate."""
        yield "", self.w_in[self.gate_at:self.gate_at + self.width]
        yield ".b", self.gate_bias

    def finalize(self) -> None:
        pass

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {}

    @property
    def state_width(self) -> int:
        return 0

    def forward(self, h: torch.Tensor, batch, cache, state, ctx: StepContext) -> tuple[torch.Tensor, ElementGate]:
        """The mixer's result and the gate it enters the stream with."""
        proj = gemm.serve_linear(h, self.w_in)
        out = torch.empty(h.shape[0], self.w_o.shape[1], dtype=h.dtype, device=h.device)
        if self.out_width < out.shape[1]:
            out[:, self.out_width:] = 0
        self.mix(proj, out, batch, cache, state, ctx)
        return gemm.serve_linear(out, self.w_o), ElementGate(proj[:, self.gate_at:self.gate_at + self.width], self.gate_bias)


class RetentionMixer(Mixer):
    """Reads q | k | v | gate."""

    def __init__(self, cfg: RetentionConfig, width: int, eps: float):
        s = cfg.shape
        super().__init__(s.proj_width, s.out_width, width, eps)
        self.cfg = cfg
        device = self.gate_bias.device
        self.register_buffer("inv_freq", rope.rope_inv_freq(s.rot, cfg.base).to(device), persistent=False)
        self.register_buffer("powers", s.powers().to(device), persistent=False)

    def tensors(self):
        """(checkpoint name under '.mix.', parameter or view of one)."""
        s = self.cfg.shape
        yield from self._rows(q=s.qk_width, k=s.qk_width, v=s.out_width, g=s.out_width)
        yield "o", self.w_o[:, :s.out_width]

    @property
    def state_width(self) -> int:
        return self.cfg.shape.state_width

    def mix(self, proj, out, batch, cache, state, ctx: StepContext) -> None:
        s = self.cfg.shape
        cs = ctx.angles((s.rot, self.cfg.base), self.inv_freq)
        recurrent.retention(proj, s, self.powers, self.eps, cs, ctx.rows, state, batch.n_single, batch.portions,
                            out[:, :s.out_width])


class AttentionMixer(Mixer):
    """Reads q | k | v | gate per element."""

    def __init__(self, cfg: AttentionConfig, width: int, eps: float):
        s = cfg.shape
        super().__init__(s.in_width + s.out_width, s.out_width, width, eps)
        self.cfg = cfg
        self.q_norm, self.k_norm, self.score_add = fp32_param(s.dim), fp32_param(s.dim), fp32_param(s.heads)
        self.register_buffer("slopes", window.distance_slopes(s.heads).to(self.q_norm.device), persistent=False)
        self.limit = math.inf                     # of a score before its temperature and bias

    def tensors(self):
        s = self.cfg.shape
        yield from self._rows(q=s.q_width, k=s.kv_heads * s.dim, v=s.kv_heads * s.vdim, g=s.out_width)
        yield "q.norm", self.q_norm
        yield "k.norm", self.k_norm
        yield "pb", self.score_add
        yield "o", self.w_o[:, :s.out_width]

    def finalize(self) -> None:
        """A normed head has at most dim in its square sum, so the norms' largest weights bound every product (2% for rounding)."""
        s = self.cfg.shape
        self.limit = 1.02 * abs(s.scale) * s.dim * float(self.q_norm.abs().max() * self.k_norm.abs().max())

    def score_bias(self, longest: int) -> ScoreBias:
        """For sequences of up to `longest` tokens; the temperature is one at the first token and moves one way from there."""
        coef, every = self.cfg.shape.temperature
        return ScoreBias(self.slopes, self.score_add, self.limit * max(1.0, abs(1.0 + coef * math.log(longest // every + 1))))

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {"kv": (self.cfg.shape.row_width,)}

    def mix(self, proj, out, batch, cache, state, ctx: StepContext) -> None:
        s, T, rows_cache = self.cfg.shape, proj.shape[0], cache["kv"]
        window.prepare(proj, s, self.q_norm, self.k_norm, self.eps, None, batch.slots, rows_cache, pos=batch.positions)
        gate, bias = proj[:, s.in_width:s.in_width + s.out_width], self.score_bias(batch.max_len)
        tensor_cores = proj.is_cuda and proj.dtype == torch.bfloat16 and window.portions_supported(s)
        nd = batch.n_single if tensor_cores else T
        if nd > 0:
            window.attend_rows(proj[:nd], s, rows_cache, batch.block_table, batch.row_seq[:nd], ctx.row_len[:nd], batch.max_len,
                               out[:nd, :s.out_width], gate=gate[:nd], bias=bias)
        if nd < T:
            keys = batch.prompt_context(s.mask)
            rows = None if keys.slots is None else latent.gather_rows(rows_cache, keys.slots)
            window.attend_portions(proj[nd:], s, rows, keys.cu_q, keys.cu_k, keys.max_q, out[nd:], gate=gate[nd:], bias=bias)


class LatentMixer(Mixer):
    """Reads q | latent | gate per head."""

    def __init__(self, cfg: LatentConfig, width: int, eps: float):
        m = cfg.shape
        super().__init__(m.q_width + m.rank + m.heads, m.heads * m.vdim, width, eps)
        self.cfg = cfg
        self.kv_norm = fp32_param(m.rank)
        self.w_kv = weight_param(m.heads * (m.dim + m.vdim), m.rank)          # keys | values, head by head
        self.register_buffer("w_uk_t", torch.empty(m.heads, m.rank, m.dim), persistent=False)
        self.register_buffer("no_freq", torch.empty(0, dtype=torch.float32), persistent=False)

    def tensors(self):
        m = self.cfg.shape
        yield from self._rows(q=m.q_width, dkv=m.rank, g=m.heads)
        yield "dkv.norm", self.kv_norm
        yield "uk", self.w_kv[:m.heads * m.dim]
        yield "uv", self.w_kv[m.heads * m.dim:]
        yield "o", self.w_o[:, :m.heads * m.vdim]

    def finalize(self) -> None:
        """The key expansion transposed per head, for queries carried into latent space."""
        m = self.cfg.shape
        self.w_uk_t.copy_(self.w_kv[:m.heads * m.dim].view(m.heads, m.dim, m.rank).transpose(1, 2))

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {"latent": (self.cfg.shape.row_width,)}

    def mix(self, proj, out, batch, cache, state, ctx: StepContext) -> None:
        m, T, rows_cache = self.cfg.shape, proj.shape[0], cache["latent"]
        expanded = proj.is_cuda and proj.dtype == torch.bfloat16 and latent.expanded_supported(m)
        nd = batch.n_single if expanded else T
        gate = proj[:, m.q_width + m.rank:m.q_width + m.rank + m.heads]
        flat = latent.prepare(proj, m, self.kv_norm, self.eps, self.no_freq, batch.positions, batch.slots, rows_cache, nd < T)
        if nd > 0:
            q = proj[:nd, :m.q_width].view(nd, m.heads, m.dim)
            o = latent.attend_latent(grouped.head_linear(q, self.w_uk_t), proj[:nd], m, rows_cache, batch.block_table,
                                     batch.row_seq[:nd], ctx.row_len[:nd], batch.max_len)
            w_uv = self.w_kv[m.heads * m.dim:].view(m.heads, m.vdim, m.rank)
            grouped.head_linear(o, w_uv, out[:nd, :m.heads * m.vdim].unflatten(1, (m.heads, m.vdim)),
                                gate[:nd, :, None].expand(-1, -1, m.vdim))
        if nd < T:
            keys = batch.prompt_context(m.mask)
            rows = flat[nd:] if keys.slots is None else latent.gather_rows(rows_cache, keys.slots)
            kv = gemm.matmul_nt(rows[:, :m.rank], self.w_kv)
            latent.attend_expanded(proj[nd:], kv, rows, m, keys.cu_q, keys.cu_k, keys.max_q, out[nd:], gate[nd:])


MIXERS = {RetentionConfig: RetentionMixer, AttentionConfig: AttentionMixer, LatentConfig: LatentMixer}


# ---------------------------------------------------------------------------------------------- feed-forward
class FeedForward(nn.Module):
    """Projection row: the inner values | padding | the residual gate | padding; the activation applies to the first two."""

    def __init__(self, width: int, ff: int):
        super().__init__()
        self.ff, self.width = ff, width
        self.inner = -(-ff // grouped.ACT_BLOCK) * grouped.ACT_BLOCK
        self.w_in, self.w_down = weight_param(up8(self.inner + width), width), weight_param(width, self.inner)
        self.gate_bias, self.act = fp32_param(width), fp32_param(2)
        self.act_args = (0.0, 0.0)                # factors of the activation's square and of its exponential part

    def tensors(self):
        yield "up", self.w_in[:self.ff]
        yield "down", self.w_down[:, :self.ff]
        yield "act", self.act

    def residual_gate(self):
        yield "", self.w_in[self.inner:self.inner + self.width]
        yield ".b", self.gate_bias

    def finalize(self) -> None:
        p, q = self.act.double().tolist()
        softplus = lambda z: max(z, 0.0) + math.log1p(math.exp(-abs(z)))     # noqa: E731
        self.act_args = softplus(p), 0.5 + softplus(q)

    def forward(self, h: torch.Tensor) -> tuple[torch.Tensor, ElementGate]:
        a, b = self.act_args
        u = gemm.serve_linear(h, self.w_in, act=grouped.ACT_XIELU, cap=a, second=b, act_cols=self.inner)
        return gemm.serve_linear(u[:, :self.inner], self.w_down), ElementGate(u[:, self.inner:self.inner + self.width], self.gate_bias)


# ---------------------------------------------------------------------------------------------- the decoder
class LovuraxLayer(nn.Module):
    def __init__(self, cfg: LovuraxConfig, index: int):
        super().__init__()
        W, l = cfg.hidden_size, cfg.layers[index]
        self.norm1 = fp32_param(W)
        self.mixer = MIXERS[type(l.mixer)](l.mixer, W, cfg.eps)
        self.ff = None
        if l.ff is not None:
            self.norm2, self.ff = fp32_param(W), FeedForward(W, l.ff)


class LovuraxForCausalLM(ServedDecoder):
    LIBRARIES = ("stream", "window", "recurrent", "retention", "latent", "latent_prefill", "skinny", "gemm")

    def __init__(self, cfg: LovuraxConfig):
        super().__init__()
        self.config = cfg
        self.embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.hidden_size), requires_grad=False)
        self.layers = nn.ModuleList(LovuraxLayer(cfg, i) for i in range(cfg.num_hidden_layers))
        self.final_norm = fp32_param(cfg.hidden_size)

    # ---------------------------------------------------------------- weights
    def _checkpoint_tensors(self):
        yield "embed", self.embed
        for i, l in enumerate(self.layers):
            for part, norm, mod, gate in (("mix", "norm1", l.mixer, "rg1"), ("mlp", "norm2", l.ff, "rg2")):
                if mod is None:
                    continue
                yield f"l{i}.{norm}", getattr(l, norm)
                for name, t in mod.tensors():
                    yield f"l{i}.{part}.{name}", t
                for name, t in mod.residual_gate():
                    yield f"l{i}.{gate}{name}", t
        yield "final.norm", self.final_norm

    @torch.no_grad()
    def reset_parameters(self, seed: int = 0) -> None:
        """Random weights from the parameters' own device generator (same device type and seed: same model)."""
        gen = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, t in self._checkpoint_tensors():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("norm1", "norm2", "norm"):
                t.fill_(1.0)
            elif leaf in ("b", "act"):
                t.zero_()
            elif leaf == "pb":
                t.fill_(RANDOM_SCORE_ADD)
            else:
                t.normal_(0.0, 1.0 / math.sqrt(t.shape[-1]), generator=gen)
        self.finalize()

    def finalize(self) -> None:
        for l in self.layers:
            l.mixer.finalize()
            if l.ff is not None:
                l.ff.finalize()

    # ---------------------------------------------------------------- serving interface of the engine
    def cache_spec(self):
        from ..inference.kv_cache import CacheSpec
        return CacheSpec([l.mixer.cache_entry() for l in self.layers], [l.mixer.state_width for l in self.layers])

    @torch.no_grad()
    def serve(self, batch, cache, observe=None) -> torch.Tensor:
        """Final-norm hidden state of the batch's wanted rows.  `observe(n, x)`: called with the stream after layer n (not
        the last)."""
        cfg, L, dtype = self.config, len(self.layers), self.embed.dtype
        ctx = StepContext(stream.StreamRows(batch.row_prev, batch.row_next), batch.positions, batch.positions + 1)
        x, h = stream.prenorm_embed(batch.token_ids, self.embed, self.layers[0].norm1, cfg.eps, 0.0)
        for i, layer in enumerate(self.layers):
            y, gate = layer.mixer(h, batch, cache.entries[i], cache.state[i], ctx)
            if layer.ff is not None:
                x, h = stream.prenorm(x, y, gate, None, layer.norm2, cfg.eps, dtype, 0.0)
                y, gate = layer.ff(h)
            if i + 1 == L:
                break
            x, h = stream.prenorm(x, y, gate, None, self.layers[i + 1].norm1, cfg.eps, dtype, 0.0)
            if observe is not None:
                observe(i, x)
        return stream.prenorm_final(x, y, gate, None, self.final_norm, cfg.eps, batch.out_rows, dtype, 0.0)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return gemm.serve_linear(hidden, self.embed, torch.float32, grouped.ACT_SCALE, self.config.logit_scale)


def build_model(config, dtype=torch.bfloat16, device=None, seed: int | None = None) -> LovuraxForCausalLM:
    """Randomly initialised model of a preset name, a config.json dictionary or a LovuraxConfig."""
    if isinstance(config, str):
        config = PRESETS[config]
    elif isinstance(config, dict):
        config = LovuraxConfig.from_dict(config)
    return LovuraxForCausalLM.random(config, dtype, device, seed)


def load_model(config: dict, state_dict: dict[str, torch.Tensor], dtype=torch.bfloat16, device=None) -> LovuraxForCausalLM:
    return LovuraxForCausalLM.from_checkpoint(LovuraxConfig.from_dict(config), state_dict, dtype, device)
