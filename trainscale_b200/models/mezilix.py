"""Mezilix: a decoder with windowed latent attention, routed squared-ReLU experts beside it (parallel block), token shift
in front of the mixer, a bigram embedding, and a depth average of all layer results after every layer.

Per layer, with X_0 the embedding and x the stream (x = X_0 before the first layer):
    h   = x / rms(x) * g                                   (g one number)
    hs  = h + (h of the token before - h) * mu
    X_n = x + latent_attention(hs) + experts(h)
    x   = sum_{j <= n} a_j X_j                             (n = number of this layer, from 1)
Everything between two GEMM groups is one launch (ops/stream.boundary); the stream, its history and the state are fp32.

A token leaves one latent row per layer in the paged cache; a sequence's state is its last token (bigram) and the last h
of every layer (token shift), kept in the cache's state slots.  `serve` runs one flattened batch of decoding rows and
portions of prompts for the engine; sizes and constants all come from the configuration and may differ per layer.
"""
from __future__ import annotations

import math
from dataclasses import dataclass
from typing import Any

import torch
import torch.nn as nn

from ..ops import gemm, grouped, latent_attention as latent, moe, rope, stream
from ..ops.latent_attention import LatentShape


@dataclass(frozen=True)
class ExpertShape:
    experts: int
    top: int
    ff: int


@dataclass(frozen=True)
class LayerConfig:
    mixer: LatentShape
    mlp: ExpertShape | None


@dataclass(frozen=True)
class MezilixConfig:
    vocab_size: int
    hidden_size: int
    eps: float
    buckets: int
    mul_prev: int
    mul_cur: int
    layers: tuple[LayerConfig, ...]

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict[str, Any]) -> "MezilixConfig":
        """Reads a config.json of this architecture."""
        layers = []
        for i, l in enumerate(d["layers"]):
            if l["type"] != "latent_attention":
                raise ValueError(f"layer {i}: unknown mixer {l['type']!r}")
            m = l["mixer"]
            if m["rot"]["dims"] != m["rot_dim"] or m["rot_dim"] % 2:
                raise ValueError(f"layer {i}: the rotation covers the whole (even) rotated part of a head")
            mixer = LatentShape(m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"], m["mask"]["size"],
                                float(m["scale"]), float(m["rot"]["base"]))
            mlp = None
            if l.get("mlp") is not None:
                f = l["mlp"]
                if f["kind"] != "moe":
                    raise ValueError(f"layer {i}: unknown feed-forward {f['kind']!r}")
                mlp = ExpertShape(f["router"]["experts"], f["router"]["top"], f["expert"]["ff"])
                if not 0 < mlp.top <= min(mlp.experts, 32) or mlp.experts > 1024:
                    raise ValueError(f"layer {i}: {mlp.top} of {mlp.experts} experts; at most 32 of 1024 are supported")
            layers.append(LayerConfig(mixer, mlp))
        bg = d["embedding"]["bigram"]
        return cls(d["vocab"], d["width"], float(d["norm"]["eps"]), bg["buckets"], bg["mul_prev"], bg["mul_cur"], tuple(layers))

    def to_dict(self) -> dict[str, Any]:
        layers = []
        for l in self.layers:
            m = l.mixer
            layers.append({
                "type": "latent_attention",
                "mixer": {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot, "vdim": m.vdim, "kv_rank": m.rank,
                          "mask": {"size": m.window}, "rot": {"base": m.rope_base, "dims": m.rot}, "scale": m.scale},
                "mlp": None if l.mlp is None else {"kind": "moe", "expert": {"ff": l.mlp.ff},
                                                   "router": {"experts": l.mlp.experts, "top": l.mlp.top}}})
        return {"architecture": "Mezilix", "vocab": self.vocab_size, "width": self.hidden_size, "norm": {"eps": self.eps},
                "embedding": {"bigram": {"buckets": self.buckets, "mul_prev": self.mul_prev, "mul_cur": self.mul_cur}},
                "layers": layers}


def uniform_config(layers: int, vocab: int, width: int, heads: int, dim: int, rot_dim: int, vdim: int, kv_rank: int,
                   window: int, experts: int, top: int, ff: int, buckets: int, rope_base: float = 10000.0,
                   mul_prev: int = 8191, mul_cur: int = 131, eps: float = 1e-5) -> MezilixConfig:
    """A configuration whose layers are all alike."""
    mixer = LatentShape(heads, dim, rot_dim, vdim, kv_rank, window, (dim + rot_dim) ** -0.5, rope_base)
    return MezilixConfig(vocab, width, eps, buckets, mul_prev, mul_cur,
                         (LayerConfig(mixer, ExpertShape(experts, top, ff)),) * layers)


PRESETS: dict[str, MezilixConfig] = {
    "mezilix-tiny": uniform_config(layers=4, vocab=32000, width=320, heads=4, dim=64, rot_dim=32, vdim=64, kv_rank=96,
                                   window=128, experts=8, top=2, ff=160, buckets=4093),
    "mezilix-4b": uniform_config(layers=16, vocab=64000, width=2048, heads=16, dim=128, rot_dim=64, vdim=128, kv_rank=512,
                                 window=1024, experts=32, top=4, ff=1536, buckets=65521, rope_base=500000.0),
}


class MezilixLayer(nn.Module):
    def __init__(self, cfg: MezilixConfig, index: int):
        super().__init__()
        W, m, f = cfg.hidden_size, cfg.layers[index].mixer, cfg.layers[index].mlp
        self.mixer, self.mlp = m, f

        def fp32(*shape):
            return nn.Parameter(torch.empty(*shape, dtype=torch.float32), requires_grad=False)

        def weight(*shape):
            return nn.Parameter(torch.empty(*shape), requires_grad=False)

        self.norm1, self.shift, self.dwa = fp32(()), fp32(W), fp32(index + 2)
        self.w_in = weight(m.q_width + m.rank + m.rot, W)                # queries | latent | shared rotated key part
        self.kv_norm = fp32(m.rank)
        self.w_kv = weight(m.heads * (m.dim + m.vdim), m.rank)           # unrotated keys | values, head by head
        self.w_o = weight(W, m.heads * m.vdim)
        if f is not None:
            self.router = weight(f.experts, W)
            self.w_up, self.w_down = weight(f.experts, f.ff, W), weight(f.experts, W, f.ff)
        self.register_buffer("w_uk_t", torch.empty(m.heads, m.rank, m.dim), persistent=False)
        self.register_buffer("inv_freq", rope.rope_inv_freq(m.rot, m.rope_base).to(self.norm1.device), persistent=False)

    @torch.no_grad()
    def finalize(self) -> None:
        """Derived weights: the key expansion transposed per head, for queries carried into latent space."""
        m = self.mixer
        self.w_uk_t.copy_(self.w_kv[:m.heads * m.dim].view(m.heads, m.dim, m.rank).transpose(1, 2))

    def mix(self, hs: torch.Tensor, batch, cache: torch.Tensor, row_len: torch.Tensor, eps: float) -> torch.Tensor:
        """Latent attention of a flattened batch: single rows in latent space, portions of prompts expanded."""
        m = self.mixer
        T = hs.shape[0]
        expanded = hs.is_cuda and hs.dtype == torch.bfloat16 and latent.expanded_supported(m)
        nd = batch.n_single if expanded else T
        proj = gemm.serve_linear(hs, self.w_in)
        flat = latent.prepare(proj, m, self.kv_norm, eps, self.inv_freq, batch.positions, batch.slots, cache, nd < T)
        out = torch.empty(T, m.heads * m.vdim, dtype=hs.dtype, device=hs.device)
        if nd > 0:
            q = proj[:nd, :m.q_width].view(nd, m.heads, m.dim + m.rot)[..., :m.dim]
            o = latent.attend_latent(grouped.head_linear(q, self.w_uk_t), proj[:nd], m, cache, batch.block_table,
                                     batch.row_seq[:nd], row_len[:nd], batch.max_len)
            w_uv = self.w_kv[m.heads * m.dim:].view(m.heads, m.vdim, m.rank)
            grouped.head_linear(o, w_uv, out[:nd].view(nd, m.heads, m.vdim))
        if nd < T:
            ctx = batch.prompt_context(m.mask)
            rows = flat[nd:] if ctx.slots is None else latent.gather_rows(cache, ctx.slots)
            kv = gemm.matmul_nt(rows[:, :m.rank], self.w_kv)
            latent.attend_expanded(proj[nd:], kv, rows, m, ctx.cu_q, ctx.cu_k, ctx.max_q, out[nd:])
        return gemm.serve_linear(out, self.w_o)

    def feed_forward(self, h: torch.Tensor):
        """Outputs of the routed experts, their rows and weights (ops/moe.routed_experts); None without experts."""
        if self.mlp is None:
            return None
        logits = gemm.serve_linear(h, self.router, torch.float32)
        return moe.routed_experts(h, logits, self.w_up, self.w_down, self.mlp.top, grouped.ACT_RELU_SQUARED)


class MezilixForCausalLM(nn.Module):
    # libraries `serve` needs (compiled together at the first use)
    LIBRARIES = ("stream", "latent", "latent_prefill", "skinny", "moe", "gemm")

    def __init__(self, cfg: MezilixConfig):
        super().__init__()
        self.config = cfg
        W = cfg.hidden_size
        self.embed = nn.Parameter(torch.empty(cfg.vocab_size, W), requires_grad=False)
        self.bigram = nn.Parameter(torch.empty(cfg.buckets + 1, W), requires_grad=False)
        self.layers = nn.ModuleList(MezilixLayer(cfg, i) for i in range(cfg.num_hidden_layers))
        self.final_norm = nn.Parameter(torch.empty((), dtype=torch.float32), requires_grad=False)
        self.head = nn.Parameter(torch.empty(cfg.vocab_size, W), requires_grad=False)
        self._side = None                 # stream of the experts in captured decode steps

    # ---------------------------------------------------------------- weights
    @torch.no_grad()
    def reset_parameters(self, seed: int = 0) -> None:
        """Random weights from the parameters' own device generator (same device type and seed: same model)."""
        gen = torch.Generator(device=self.embed.device).manual_seed(seed)
        for name, p in self.named_parameters():
            if name.endswith(("norm1", "kv_norm", "final_norm")):
                p.fill_(1.0)
            elif name.endswith("shift"):
                p.uniform_(0.0, 1.0, generator=gen)
            elif name.endswith("dwa"):
                p.normal_(0.0, 0.1, generator=gen)
                p[-1] = 1.0
            else:
                p.normal_(0.0, 1.0 if name in ("embed", "bigram") else 1.0 / math.sqrt(p.shape[-1]), generator=gen)
        for l in self.layers:
            l.finalize()

    def _checkpoint_tensors(self):
        """(checkpoint name, parameter or view of one) of every stored tensor."""
        yield "embed", self.embed
        yield "bigram", self.bigram
        for i, l in enumerate(self.layers):
            m, p = l.mixer, f"l{i}."
            yield p + "norm1", l.norm1
            yield p + "shift", l.shift
            yield p + "dwa", l.dwa
            yield p + "mix.q", l.w_in[:m.q_width]
            yield p + "mix.dkv", l.w_in[m.q_width:]
            yield p + "mix.dkv.norm", l.kv_norm
            yield p + "mix.uk", l.w_kv[:m.heads * m.dim]
            yield p + "mix.uv", l.w_kv[m.heads * m.dim:]
            yield p + "mix.o", l.w_o
            if l.mlp is not None:
                yield p + "mlp.router", l.router
                for e in range(l.mlp.experts):
                    yield f"{p}mlp.e{e}.up", l.w_up[e]
                    yield f"{p}mlp.e{e}.down", l.w_down[e]
        yield "final.norm", self.final_norm
        yield "head", self.head

    @torch.no_grad()
    def load_checkpoint(self, sd: dict[str, torch.Tensor]) -> None:
        want = dict(self._checkpoint_tensors())
        missing, extra = sorted(want.keys() - sd.keys()), sorted(sd.keys() - want.keys())
        if missing or extra:
            raise KeyError(f"checkpoint does not fit the configuration: missing {missing[:6]}, unknown {extra[:6]}")
        for name, dst in want.items():
            if tuple(sd[name].shape) != tuple(dst.shape):
                raise ValueError(f"{name}: shape {tuple(sd[name].shape)}, the configuration says {tuple(dst.shape)}")
            dst.copy_(sd[name])
        for l in self.layers:
            l.finalize()

    @torch.no_grad()
    def to_checkpoint(self) -> dict[str, torch.Tensor]:
        return {name: t.detach().to(torch.bfloat16) for name, t in self._checkpoint_tensors()}

    # ---------------------------------------------------------------- serving interface of the engine
    def cache_spec(self):
        from ..inference.kv_cache import CacheSpec
        return CacheSpec([{"latent": (l.mixer.row_width,)} for l in self.layers],
                         [self.config.hidden_size] * len(self.layers))

    def _side_stream(self) -> "torch.cuda.Stream":
        if self._side is None:
            self._side = torch.cuda.Stream(device=self.embed.device)
        return self._side

    @torch.no_grad()
    def serve(self, batch, cache, observe=None) -> torch.Tensor:
        """Final-norm hidden state of the batch's wanted rows.  `observe(n, x)`: called with the stream after layer n."""
        cfg, L = self.config, len(self.layers)
        T, dtype, dev = batch.num_tokens, self.embed.dtype, self.embed.device
        hist = torch.empty(L + 1, T, cfg.hidden_size, dtype=torch.float32, device=dev)
        rows = stream.StreamRows(batch.row_prev, batch.row_next)
        row_len = batch.positions + 1
        first = self.layers[0]
        h, hs = stream.embed(batch.token_ids, batch.prev_tokens, self.embed, self.bigram, cfg.mul_prev, cfg.mul_cur, hist,
                             first.norm1, cfg.eps, first.shift, rows, cache.state[0])
        x = hist[0]
        for i, layer in enumerate(self.layers):
            if batch.captured and layer.mlp is not None:
                # a decode step is a chain of short kernels: mixer and experts of the parallel block run side by side
                main, side = torch.cuda.current_stream(), self._side_stream()
                side.wait_stream(main)
                with torch.cuda.stream(side):
                    experts = layer.feed_forward(h)
                mixer = layer.mix(hs, batch, cache.entries[i]["latent"], row_len, cfg.eps)
                main.wait_stream(side)
            else:
                mixer = layer.mix(hs, batch, cache.entries[i]["latent"], row_len, cfg.eps)
                experts = layer.feed_forward(h)
            if i + 1 == L:
                break
            nxt = self.layers[i + 1]
            x, h, hs = stream.boundary(x, mixer, experts, hist, layer.dwa, i + 1, nxt.norm1, cfg.eps, nxt.shift, rows,
                                       cache.state[i + 1], dtype)
            if observe is not None:
                observe(i, x)
        return stream.final(x, mixer, experts, hist, self.layers[-1].dwa, L, self.final_norm, cfg.eps, batch.out_rows, dtype)

    def logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return gemm.serve_linear(hidden, self.head, torch.float32)

    @torch.no_grad()
    def forward(self, input_ids: torch.Tensor) -> torch.Tensor:
        """fp32 logits [B, S, vocab] of whole sequences (a throw-away cache; inference only)."""
        from ..inference.batch import HostBatch, StepEntry
        from ..inference.kv_cache import PagedKVCache
        B, S = input_ids.shape
        bs = 64
        cache = PagedKVCache(len(self.layers), B * -(-S // bs), bs, dtype=self.embed.dtype, device=self.embed.device,
                             spec=self.cache_spec(), state_slots=B)
        host = HostBatch(cache, [StepEntry(b, row, list(range(S))) for b, row in enumerate(input_ids.tolist())])
        return self.logits(self.serve(host.to_device(self.embed.device), cache)).view(B, S, -1)


def build_model(config, dtype=torch.bfloat16, device=None, seed: int | None = None) -> MezilixForCausalLM:
    """Randomly initialised model of a preset name, a config.json dictionary or a MezilixConfig."""
    model = _empty(config, dtype, device)
    model.reset_parameters(0 if seed is None else seed)
    return model


def _empty(config, dtype, device) -> MezilixForCausalLM:
    if isinstance(config, str):
        config = PRESETS[config]
    elif isinstance(config, dict):
        config = MezilixConfig.from_dict(config)
    device = torch.device(device or "cpu")
    if device.type == "cuda":
        from ..ops import _lib
        _lib.prepare(list(MezilixForCausalLM.LIBRARIES))
    prev = torch.get_default_dtype()
    torch.set_default_dtype(dtype)
    try:
        with torch.device(device):
            return MezilixForCausalLM(config).eval()
    finally:
        torch.set_default_dtype(prev)


def load_model(config: dict, state_dict: dict[str, torch.Tensor], dtype=torch.bfloat16, device=None) -> MezilixForCausalLM:
    model = _empty(config, dtype, device)
    model.load_checkpoint(state_dict)
    return model
