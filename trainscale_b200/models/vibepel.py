"""Vibepel: a decoder that norms every sublayer's OUTPUT (x + norm(f(x))), with layers of two kinds: sliding-window attention
and a gated delta rule side by side, or WKV time mixing; dense squared-ReLU feed-forwards; tied embedding and soft-capped
logits.

    x <- x + n1(mixer(x)),  x <- x + n2(W_down relu(W_up x)^2),   n(y) = y / rms(y) * (1 + w)
    parallel mixer:  left_scale * attention(x) + right_scale * delta(x), one input and one output projection for both
    WKV mixer:       r, k, v, gate and decay each read their own mix of x and the previous token's x
The residual sum between two sublayers, its norm, the cast for the next GEMM or the token-shift mixes of a WKV layer are one
launch (ops/stream.postnorm); the stream and all recurrent state are fp32.

A token leaves one row of keys and values per parallel layer in the paged cache.  A sequence's state rows hold the last
convolution inputs and the delta rule's matrices, or the last x and the WKV matrices.  `serve` runs one flattened batch of
decoding rows and portions of prompts for the engine; sizes and constants come from the configuration and may differ per
layer (the inner size of the WKV decay from its tensor).
"""
from __future__ import annotations

import math
from dataclasses import dataclass, field
from typing import Any

import torch
import torch.nn as nn

from ..ops import gemm, grouped, latent_attention as latent, recurrent, rope, stream, window_attention as window
from ..ops.recurrent import DeltaShape, DeltaWeights, WkvShape, WkvWeights
from ..ops.window_attention import WindowShape
from .served import ServedDecoder, fp32_param, require, up8, weight_param

SHIFTS = "rkvgw"            # inputs of a WKV mixer, in the order of its mixes


@dataclass(frozen=True)
class Rotation:
    dims: int
    base: float
    # wavelengths above original / low are slowed down by `factor`, below original / high kept, linear in between
    scaling: tuple[float, float, float, float] | None = None      # factor, low, high, original

    def inv_freq(self) -> torch.Tensor:
        if self.scaling is None:
            return rope.rope_inv_freq(self.dims, self.base)
        factor, low, high, original = self.scaling
        return rope.rope_inv_freq(self.dims, self.base, "llama3", factor=factor, low_freq_factor=low, high_freq_factor=high,
                                  original_max_pos=original)


@dataclass(frozen=True)
class ParallelConfig:
    left: WindowShape
    rot: Rotation
    right: DeltaShape
    left_scale: float
    right_scale: float


@dataclass(frozen=True)
class WkvConfig:
    shape: WkvShape
    decay_rank: int           # inner size of the decay's two projections


@dataclass(frozen=True)
class LayerConfig:
    mixer: ParallelConfig | WkvConfig
    ff: int | None


@dataclass(frozen=True)
class VibepelConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    embed_scale: float
    logit_softcap: float
    layers: tuple[LayerConfig, ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict[str, Any], shapes: dict[str, tuple[int, ...]] | None = None) -> "VibepelConfig":
        """Reads a config.json of this architecture.  `shapes`: of the checkpoint's tensors, for the size that the file
        leaves to them (else `decay_rank` of a WKV mixer, 32 by default)."""
        W = d["width"]
        layers = []
        for i, l in enumerate(d["layers"]):
            m = l["mixer"]
            if l["type"] == "wkv":
                w1 = (shapes or {}).get(f"l{i}.mix.w1")
                mixer = WkvConfig(WkvShape(m["heads"], m["dim"], W), w1[0] if w1 else m.get("decay_rank", 32))
                require(m["dim"] <= recurrent.MAX_HEAD, i, f"WKV heads of up to {recurrent.MAX_HEAD} dimensions")
            elif l["type"] == "parallel":
                a, b, r = m["left"], m["right"], m["left"]["rot"]
                s = r.get("scaling")
                rot = Rotation(r["dims"], float(r["base"]),
                               None if not s else tuple(float(s[k]) for k in ("factor", "low", "high", "original")))
                mixer = ParallelConfig(
                    WindowShape(a["heads"], a["kv_heads"], a["dim"], a["vdim"], rot.dims, a["mask"]["size"], float(a["scale"])),
                    rot, DeltaShape(b["heads"], b["kv_heads"], b["dim"], b["vdim"], b["conv"]),
                    float(m["left_scale"]), float(m["right_scale"]))
                require(rot.dims % 2 == 0 and rot.dims <= a["dim"], i, "an even number of rotated dimensions inside a head")
                require(a["heads"] % a["kv_heads"] == 0 and b["heads"] % b["kv_heads"] == 0, i, "whole head groups")
                require(a["mask"]["size"] > 0 and b["conv"] > 0, i, "a window and a convolution of at least one token")
                require(max(b["dim"], b["vdim"]) <= recurrent.MAX_HEAD, i,
                        f"delta rule heads of up to {recurrent.MAX_HEAD} dimensions")
            else:
                raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
            f = l.get("mlp")
            if f is not None and f["kind"] != "dense":
                raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
            layers.append(LayerConfig(mixer, None if f is None else f["ff"]))
        if not layers:
            raise ValueError("a model needs layers")
        return cls(d["vocab"], W, float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["logit_softcap"]), tuple(layers))

    def to_dict(self) -> dict[str, Any]:
        layers = []
        for l in self.layers:
            if isinstance(l.mixer, WkvConfig):
                kind, s = "wkv", l.mixer.shape
                mixer: dict[str, Any] = {"heads": s.heads, "dim": s.dim, "decay_rank": l.mixer.decay_rank}
            else:
                kind, a, b, r = "parallel", l.mixer.left, l.mixer.right, l.mixer.rot
                rot: dict[str, Any] = {"base": r.base, "dims": r.dims}
                if r.scaling is not None:
                    rot["scaling"] = dict(zip(("factor", "low", "high", "original"), r.scaling))
                mixer = {"left": {"heads": a.heads, "kv_heads": a.kv_heads, "dim": a.dim, "vdim": a.vdim, "scale": a.scale,
                                  "mask": {"size": a.window}, "rot": rot},
                         "right": {"heads": b.heads, "kv_heads": b.kv_heads, "dim": b.dim, "vdim": b.vdim, "conv": b.taps},
                         "left_scale": l.mixer.left_scale, "right_scale": l.mixer.right_scale}
            layers.append({"type": kind, "mixer": mixer, "mlp": None if l.ff is None else {"kind": "dense", "ff": l.ff}})
        return {"architecture": "Vibepel", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "logit_softcap": self.logit_softcap, "layers": layers}


def pattern_config(layers: int, vocab: int, width: int, heads: int, kv_heads: int, dim: int, window: int, ff: int,
                   delta_heads: int, delta_kv_heads: int, delta_dim: int, delta_vdim: int, wkv_heads: int, wkv_dim: int,
                   wkv_every: int = 4, taps: int = 4, rot_dims: int | None = None, rope_base: float = 10000.0,
                   decay_rank: int = 64, eps: float = 1e-6, softcap: float = 30.0) -> VibepelConfig:
    """Every `wkv_every`-th layer mixes with WKV, the others with attention and delta rule in parallel."""
    par = ParallelConfig(WindowShape(heads, kv_heads, dim, dim, rot_dims or dim, window, dim ** -0.5),
                         Rotation(rot_dims or dim, rope_base), DeltaShape(delta_heads, delta_kv_heads, delta_dim, delta_vdim, taps),
                         1.0, 1.0)
    wkv = WkvConfig(WkvShape(wkv_heads, wkv_dim, width), decay_rank)
    return VibepelConfig(vocab, width, eps, width ** 0.5, softcap,
                         tuple(LayerConfig(wkv if (i + 1) % wkv_every == 0 else par, ff) for i in range(layers)))


PRESETS: dict[str, VibepelConfig] = {
    "vibepel-tiny": pattern_config(layers=4, vocab=32000, width=320, heads=4, kv_heads=2, dim=64, window=128, ff=640,
                                   delta_heads=4, delta_kv_heads=2, delta_dim=64, delta_vdim=64, wkv_heads=5, wkv_dim=64,
                                   rot_dims=32),
    "vibepel-2b": pattern_config(layers=24, vocab=64000, width=2048, heads=16, kv_heads=4, dim=128, window=1024, ff=8192,
                                 delta_heads=16, delta_kv_heads=8, delta_dim=128, delta_vdim=128, wkv_heads=32, wkv_dim=64,
                                 rot_dims=64, rope_base=500000.0),
}


@dataclass
class StepContext:
    """What the layers of one step share."""
    rows: stream.StreamRows
    positions: torch.Tensor
    row_len: torch.Tensor                       # keys of a row before the window is applied
    side: "torch.cuda.Stream | None"            # captured decode: stream of the second mixer of a parallel layer
    _angles: dict[Rotation, torch.Tensor] = field(default_factory=dict)

    def angles(self, rot: Rotation, inv_freq: torch.Tensor) -> torch.Tensor:
        if rot not in self._angles:
            self._angles[rot] = window.angles(inv_freq, self.positions)
        return self._angles[rot]


class ParallelMixer(nn.Module):
    """Windowed attention (left) and gated delta rule (right) on the same input; projection row:
    left q | k | v | right q | k | v | gate | beta | decay."""
    mu = None                       # reads x itself

    def __init__(self, cfg: ParallelConfig, width: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        a, b = cfg.left, cfg.right
        self.right_at = a.q_width + a.kv_width
        self.w_in = weight_param(up8(self.right_at + b.proj_width), width)
        self.w_o = weight_param(width, up8(a.out_width + b.out_width))
        self.q_norm, self.k_norm = fp32_param(a.dim), fp32_param(a.dim)
        self.conv, self.A_log, self.dt_bias, self.norm = fp32_param(b.channels, b.taps), fp32_param(b.heads), fp32_param(b.heads), fp32_param(b.vdim)
        self.register_buffer("inv_freq", cfg.rot.inv_freq().to(self.q_norm.device), persistent=False)

    def tensors(self):
        """(checkpoint name under '.mix.', parameter or view of one)."""
        a, b = self.cfg.left, self.cfg.right
        kw, vw = b.kv_heads * b.dim, b.heads * b.vdim
        at = 0
        for name, n in (("left.q", a.q_width), ("left.k", a.kv_heads * a.dim), ("left.v", a.kv_heads * a.vdim),
                        ("right.q", kw), ("right.k", kw), ("right.v", vw), ("right.g", vw), ("right.b", b.heads),
                        ("right.a", b.heads)):
            yield name, self.w_in[at:at + n]
            at += n
        yield "left.q.norm", self.q_norm
        yield "left.k.norm", self.k_norm
        yield "left.o", self.w_o[:, :a.out_width]
        yield "right.o", self.w_o[:, a.out_width:a.out_width + b.out_width]
        yield "right.q.conv", self.conv[:kw]
        yield "right.k.conv", self.conv[kw:2 * kw]
        yield "right.v.conv", self.conv[2 * kw:]
        yield "right.A_log", self.A_log
        yield "right.dt_bias", self.dt_bias
        yield "right.norm", self.norm

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {"kv": (self.cfg.left.row_width,)}

    @property
    def state_width(self) -> int:
        return self.cfg.right.state_width

    def _attend(self, proj: torch.Tensor, out: torch.Tensor, batch, cache: torch.Tensor, ctx: "StepContext") -> None:
        s, T = self.cfg.left, proj.shape[0]
        tensor_cores = proj.is_cuda and proj.dtype == torch.bfloat16 and window.portions_supported(s)
        nd = batch.n_single if tensor_cores else T
        window.prepare(proj, s, self.q_norm, self.k_norm, self.eps, ctx.angles(self.cfg.rot, self.inv_freq), batch.slots, cache)
        if nd > 0:
            window.attend_rows(proj[:nd], s, cache, batch.block_table, batch.row_seq[:nd], ctx.row_len[:nd], batch.max_len, out[:nd],
                               self.cfg.left_scale)
        if nd < T:
            keys = batch.prompt_context(s.mask)
            rows = None if keys.slots is None else latent.gather_rows(cache, keys.slots)
            window.attend_portions(proj[nd:], s, rows, keys.cu_q, keys.cu_k, keys.max_q, out[nd:], self.cfg.left_scale)

    def forward(self, h: torch.Tensor, batch, cache, state: torch.Tensor, ctx: "StepContext") -> torch.Tensor:
        a, b = self.cfg.left, self.cfg.right
        T, used = h.shape[0], a.out_width + b.out_width
        proj = gemm.serve_linear(h, self.w_in)
        both = torch.empty(T, self.w_o.shape[1], dtype=h.dtype, device=h.device)
        if used < both.shape[1]:
            both[:, used:] = 0

        def right():
            recurrent.delta_rule(proj[:, self.right_at:], b, DeltaWeights(self.conv, self.A_log, self.dt_bias, self.norm),
                                 self.eps, ctx.rows, state, batch.n_single, batch.portions,
                                 both[:, a.out_width:used], self.cfg.right_scale)

        if ctx.side is not None:    # a captured decode step is a chain of short kernels: both mixers at once
            main = torch.cuda.current_stream()
            ctx.side.wait_stream(main)
            with torch.cuda.stream(ctx.side):
                right()
            self._attend(proj, both[:, :a.out_width], batch, cache["kv"], ctx)
            main.wait_stream(ctx.side)
        else:
            self._attend(proj, both[:, :a.out_width], batch, cache["kv"], ctx)
            right()
        return gemm.serve_linear(both, self.w_o)


class WkvMixer(nn.Module):
    def __init__(self, cfg: WkvConfig, width: int, eps: float):
        super().__init__()
        self.cfg, self.eps = cfg, eps
        s = cfg.shape
        self.mu = fp32_param(len(SHIFTS), width)
        self.w_rkvg = weight_param(4, s.inner, width)
        self.w1, self.w2 = weight_param(cfg.decay_rank, width), weight_param(s.inner, cfg.decay_rank)
        self.w_o = weight_param(width, s.inner)
        self.w0, self.u, self.norm = fp32_param(s.inner), fp32_param(s.heads, s.dim), fp32_param(s.inner)

    def tensors(self):
        for i, name in enumerate(SHIFTS):
            yield f"mu.{name}", self.mu[i]
        for i, name in enumerate("rkvg"):
            yield name, self.w_rkvg[i]
        for name in ("w1", "w2", "w0", "u", "norm"):
            yield name, getattr(self, name)
        yield "o", self.w_o

    def cache_entry(self) -> dict[str, tuple[int, ...]]:
        return {}

    @property
    def state_width(self) -> int:
        return self.cfg.shape.state_width

    def forward(self, mixes: torch.Tensor, batch, cache, state: torch.Tensor, ctx: "StepContext") -> torch.Tensor:
        s, T = self.cfg.shape, mixes.shape[0]
        rkvg = torch.empty(T, 4, s.inner, dtype=mixes.dtype, device=mixes.device)
        if mixes.is_cuda and gemm.few_rows(T, 4 * s.inner, mixes.shape[2]):
            grouped.head_linear(mixes[:, :4], self.w_rkvg, rkvg)
        else:
            for i in range(4):
                gemm.serve_linear(mixes[:, i], self.w_rkvg[i], out=rkvg[:, i])
        inner = gemm.serve_linear(mixes[:, 4], self.w1, act=grouped.ACT_TANH)
        w_raw = gemm.serve_linear(inner, self.w2, torch.float32)
        out = torch.empty(T, s.inner, dtype=mixes.dtype, device=mixes.device)
        recurrent.wkv(rkvg, w_raw, s, WkvWeights(self.w0, self.u, self.norm), self.eps, ctx.rows, state, batch.n_single,
                      batch.portions, out)
        return gemm.serve_linear(out, self.w_o)


class VibepelLayer(nn.Module):
    def __init__(self, cfg: VibepelConfig, index: int):
        super().__init__()
        W, l = cfg.hidden_size, cfg.layers[index]
        self.mixer = (WkvMixer if isinstance(l.mixer, WkvConfig) else ParallelMixer)(l.mixer, W, cfg.eps)
        self.norm1 = fp32_param(W)
        self.ff = l.ff
        if l.ff is not None:
            self.norm2, self.w_up, self.w_down = fp32_param(W), weight_param(l.ff, W), weight_param(W, l.ff)

    def feed_forward(self, h: torch.Tensor) -> torch.Tensor:
        return gemm.serve_linear(gemm.serve_linear(h, self.w_up, act=grouped.ACT_RELU_SQUARED), self.w_down)


class VibepelForCausalLM(ServedDecoder):
    LIBRARIES = ("stream", "window", "recurrent", "latent", "latent_prefill", "skinny", "gemm")

    def __init__(self, cfg: VibepelConfig):
        super().__init__()
        self.config = cfg
        self.embed = nn.Parameter(torch.empty(cfg.vocab_size, cfg.hidden_size), requires_grad=False)
        self.layers = nn.ModuleList(VibepelLayer(cfg, i) for i in range(cfg.num_hidden_layers))
        self.final_norm = fp32_param(cfg.hidden_size)

    # ---------------------------------------------------------------- weights
    def _checkpoint_tensors(self):
        """(checkpoint name, parameter or view of one) of every stored tensor."""
        yield "embed", self.embed
        for i, l in enumerate(self.layers):
            yield f"l{i}.norm1", l.norm1
            for name, t in l.mixer.tensors():
                yield f"l{i}.mix.{name}", t
            if l.ff is not None:
                yield f"l{i}.norm2", l.norm2
                yield f"l{i}.mlp.up", l.w_up
                yield f"l{i}.mlp.down", l.w_down
        yield "final.norm", self.final_norm

    @torch.no_grad()
    def reset_parameters(self, seed: int = 0) -> None:
        """Random weights from the parameters' own device generator (same device type and seed: same model)."""
        gen = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, p in self._checkpoint_tensors():
            leaf = name.rsplit(".", 1)[-1]
            if leaf in ("norm1", "norm2") or name == "final.norm":
                p.zero_()
            elif leaf == "norm":
                p.fill_(1.0)
            elif ".mu." in name:
                p.uniform_(0.0, 1.0, generator=gen)
            elif leaf == "A_log":
                p.uniform_(0.0, 2.0, generator=gen)
            elif leaf == "dt_bias":
                p.uniform_(-5.0, -2.0, generator=gen)
            elif leaf == "w0":
                p.uniform_(-6.0, -1.0, generator=gen)
            elif leaf == "embed":
                p.normal_(0.0, 1.0 / math.sqrt(p.shape[-1]), generator=gen)
            else:
                p.normal_(0.0, 0.5 if leaf in ("u", "conv") else 1.0 / math.sqrt(p.shape[-1]), generator=gen)

    # ---------------------------------------------------------------- serving interface of the engine
    def cache_spec(self):
        from ..inference.kv_cache import CacheSpec
        return CacheSpec([l.mixer.cache_entry() for l in self.layers], [l.mixer.state_width for l in self.layers])

    @torch.no_grad()
    def serve(self, batch, cache, observe=None) -> torch.Tensor:
        """Final-norm hidden state of the batch's wanted rows.  `observe(n, x)`: called with the stream after layer n (not
        the last)."""
        cfg, L, dtype = self.config, len(self.layers), self.embed.dtype
        rows = stream.StreamRows(batch.row_prev, batch.row_next)
        ctx = StepContext(rows, batch.positions, batch.positions + 1, self._side_stream() if batch.captured else None)
        x, h = stream.scaled_embed(batch.token_ids, self.embed, cfg.embed_scale, self.layers[0].mixer.mu, rows, cache.state[0])
        for i, layer in enumerate(self.layers):
            y = layer.mixer(h, batch, cache.entries[i], cache.state[i], ctx)
            norm = layer.norm1
            if layer.ff is not None:
                x, h = stream.postnorm(x, y, norm, cfg.eps, None, rows, None, dtype)
                y, norm = layer.feed_forward(h), layer.norm2
            if i + 1 == L:
                break
            x, h = stream.postnorm(x, y, norm, cfg.eps, self.layers[i + 1].mixer.mu, rows, cache.state[i + 1], dtype)
            if observe is not None:
                observe(i, x)
        return stream.postnorm_final(x, y, norm, self.final_norm, cfg.eps, batch.out_rows, dtype)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return gemm.serve_linear(hidden, self.embed, torch.float32, grouped.ACT_SOFTCAP, self.config.logit_softcap)


def build_model(config, dtype=torch.bfloat16, device=None, seed: int | None = None) -> VibepelForCausalLM:
    """Randomly initialised model of a preset name, a config.json dictionary or a VibepelConfig."""
    if isinstance(config, str):
        config = PRESETS[config]
    elif isinstance(config, dict):
        config = VibepelConfig.from_dict(config)
    return VibepelForCausalLM.random(config, dtype, device, seed)


def load_model(config: dict, state_dict: dict[str, torch.Tensor], dtype=torch.bfloat16, device=None) -> VibepelForCausalLM:
    return VibepelForCausalLM.from_checkpoint(VibepelConfig.from_dict(config, {k: tuple(v.shape) for k, v in state_dict.items()}), state_dict, dtype, device)
