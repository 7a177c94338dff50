"""Prefill and decode throughput of a served design beside the framework's closest existing model at equal size, with the
device time of every op and its distance from the roofline (`bench.py --serve`, `--serve-model`).

Both models run through `ModelRunner` on the engine's cache with random weights and random tokens.  Step times are CUDA
events around whole steps; for the per-op table the host first queues a spin kernel, so that a whole step is enqueued
before the device starts it and the events around each op see no launch gaps.
"""
from __future__ import annotations

import json
import math
import statistics
from dataclasses import dataclass
from pathlib import Path
from typing import Callable

import torch

from ..ops.masks import UNBOUNDED, KeyMask
from .batch import HostBatch, StepEntry
from .engine import EngineConfig, EngineCore

# name -> sizes shared by both models; Mezilix experts have two matrices of `ff`, the gated ones three of 2/3 ff
SIZES = {
    "1k": dict(layers=12, width=1024, heads=8, dim=64, rot=32, vdim=64, rank=256, window=512, experts=16, top=2, ff=1536),
    "2k": dict(layers=16, width=2048, heads=16, dim=128, rot=64, vdim=128, rank=512, window=1024, experts=32, top=4, ff=1536),
    "4k": dict(layers=8, width=4096, heads=32, dim=128, rot=64, vdim=128, rank=512, window=4096, experts=64, top=6, ff=1536),
}
# every fourth layer mixes with WKV, the others with attention and the delta rule in parallel; the closest model has gated
# feed-forwards of 2/3 ff and the attention of `heads` / `kv` in every layer
VIBEPEL_SIZES = {
    "1k": dict(layers=12, width=1024, heads=8, kv=2, dim=128, window=512, ff=4096, dheads=8, dkv=4, ddim=128, wheads=16, wdim=64),
    "2k": dict(layers=16, width=2048, heads=16, kv=4, dim=128, window=1024, ff=8192, dheads=16, dkv=8, ddim=128, wheads=32, wdim=64),
    "4k": dict(layers=8, width=4096, heads=32, kv=8, dim=128, window=4096, ff=16384, dheads=32, dkv=16, ddim=128, wheads=64, wdim=64),
}
# layers take turns: window with sinks, chunks, latent, window with sinks; the first feeds forward densely, the others through
# experts and a shared one; the closest model has the same routed experts and the attention of `heads` / `kv` in every layer
KABULIX_SIZES = {
    "1k": dict(layers=12, width=1024, heads=8, kv=2, dim=128, window=512, keep=4, chunk=1536, ldim=64, lrot=32, lvdim=64, rank=256,
               experts=16, top=2, groups=4, kept=2, ff=1536),
    "2k": dict(layers=16, width=2048, heads=16, kv=4, dim=128, window=1024, keep=4, chunk=3072, ldim=128, lrot=64, lvdim=128, rank=512,
               experts=32, top=4, groups=8, kept=4, ff=1536),
    "4k": dict(layers=8, width=4096, heads=32, kv=8, dim=128, window=4096, keep=4, chunk=4096, ldim=128, lrot=64, lvdim=128, rank=512,
               experts=64, top=6, groups=8, kept=4, ff=1536),
}
# layers take turns: retention, sigmoid attention, retention, latent attention
LOVURAX_SIZES = {
    "1k": dict(layers=12, width=1024, heads=8, kv=2, dim=128, rheads=4, rdim=128, rvdim=256, ldim=64, lvdim=64, rank=256, ff=4096),
    "2k": dict(layers=16, width=2048, heads=16, kv=4, dim=128, rheads=8, rdim=128, rvdim=256, ldim=128, lvdim=128, rank=512, ff=8192),
    "4k": dict(layers=8, width=4096, heads=32, kv=8, dim=128, rheads=16, rdim=128, rvdim=256, ldim=128, lvdim=128, rank=512, ff=16384),
}
VOCAB = 32000
FP32_TFLOPS = 74.4            # nominal: 148 SMs x 128 lanes x 2 x 1.965 GHz


def build_mezilix(z: dict):
    from ..models.mezilix import build_model, uniform_config
    return build_model(uniform_config(layers=z["layers"], vocab=VOCAB, width=z["width"], heads=z["heads"], dim=z["dim"],
                                      rot_dim=z["rot"], vdim=z["vdim"], kv_rank=z["rank"], window=z["window"],
                                      experts=z["experts"], top=z["top"], ff=z["ff"], buckets=65521),
                       torch.bfloat16, "cuda", seed=0)


def build_closest(z: dict):
    """Llama decoder with a mixture of gated experts: same width, depth, heads, experts and expert weights."""
    from ..models.llama import LlamaConfig, build_model
    cfg = LlamaConfig(vocab_size=VOCAB, hidden_size=z["width"], intermediate_size=z["ff"] * 2 // 3,
                      num_hidden_layers=z["layers"], num_attention_heads=z["heads"],
                      num_key_value_heads=z.get("kv") or max(1, z["heads"] // 4),
                      head_dim=z.get("vdim") or z["dim"], num_local_experts=z["experts"], num_experts_per_tok=z["top"],
                      model_type="mixtral", max_position_embeddings=16384)
    return build_model(cfg, torch.bfloat16, "cuda", seed=0, init_on_device=True)


def build_vibepel(z: dict):
    from ..models.vibepel import build_model, pattern_config
    return build_model(pattern_config(layers=z["layers"], vocab=VOCAB, width=z["width"], heads=z["heads"], kv_heads=z["kv"],
                                      dim=z["dim"], window=z["window"], ff=z["ff"], delta_heads=z["dheads"],
                                      delta_kv_heads=z["dkv"], delta_dim=z["ddim"], delta_vdim=z["ddim"],
                                      wkv_heads=z["wheads"], wkv_dim=z["wdim"], rot_dims=z["dim"] // 2),
                       torch.bfloat16, "cuda", seed=0)


def build_closest_dense(z: dict):
    """Llama decoder with dense gated feed-forwards: same width, depth, attention heads and feed-forward weights."""
    from ..models.llama import LlamaConfig, build_model
    cfg = LlamaConfig(vocab_size=VOCAB, hidden_size=z["width"], intermediate_size=-(-z["ff"] * 2 // 3 // 64) * 64,
                      num_hidden_layers=z["layers"], num_attention_heads=z["heads"], num_key_value_heads=z["kv"],
                      head_dim=z["dim"], max_position_embeddings=16384, tie_word_embeddings=True)
    return build_model(cfg, torch.bfloat16, "cuda", seed=0, init_on_device=True)


def build_kabulix(z: dict):
    from ..models.kabulix import build_model, pattern_config
    ff = z["ff"] * 2 // 3                    # three matrices per expert
    kinds = ("wclw" * z["layers"])[:z["layers"]]
    return build_model(pattern_config(kinds, vocab=VOCAB, width=z["width"], heads=z["heads"], kv_heads=z["kv"], dim=z["dim"],
                                      window=z["window"], keep=z["keep"], chunk=z["chunk"], latent_dim=z["ldim"],
                                      latent_rot=z["lrot"], latent_vdim=z["lvdim"], rank=z["rank"], latent_window=z["window"],
                                      ff=ff * (z["top"] + 1), experts=z["experts"], top=z["top"], expert_ff=ff, shared_ff=ff,
                                      groups=z["groups"], keep_groups=z["kept"], rot_dims=z["dim"] // 2),
                       torch.bfloat16, "cuda", seed=0)


def build_lovurax(z: dict):
    from ..models.lovurax import build_model, pattern_config
    kinds = ("rarl" * z["layers"])[:z["layers"]]
    return build_model(pattern_config(kinds, vocab=VOCAB, width=z["width"], heads=z["heads"], kv_heads=z["kv"], dim=z["dim"],
                                      ret_heads=z["rheads"], ret_dim=z["rdim"], ret_vdim=z["rvdim"], latent_dim=z["ldim"],
                                      latent_vdim=z["lvdim"], rank=z["rank"], ff=z["ff"]),
                       torch.bfloat16, "cuda", seed=0)


def make_core(model, tokens: int, seqs: int) -> EngineCore:
    cfg = EngineConfig(model="custom", tokenizer="byte", device="cuda", enforce_eager=False)
    cfg.cache.num_gpu_blocks = tokens // cfg.cache.block_size + seqs
    cfg.cache.enable_prefix_caching = False
    cfg.scheduler.max_num_seqs = seqs
    return EngineCore(cfg, model=model)


def _tokens(n: int, seed: int) -> list[int]:
    return torch.randint(0, VOCAB, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _timed(fn, n: int, warm: int = 3) -> float:
    """Median device time (ms) of `fn`, the L2 flushed between calls."""
    flush = torch.empty(64 << 20, dtype=torch.float32, device="cuda")
    out = []
    for i in range(warm + n):
        flush.zero_()
        torch.cuda._sleep(20_000_000)       # the step is enqueued while the device spins
        a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
        a.record()
        fn()
        b.record()
        b.synchronize()
        if i >= warm:
            out.append(a.elapsed_time(b))
    return statistics.median(out)


# ---------------------------------------------------------------------------------------------- per-op costs
def _bytes(*ts) -> int:
    return sum(t.numel() * t.element_size() for t in ts if isinstance(t, torch.Tensor))


class OpTimer:
    """Events around every call of the wrapped op functions; `cost(args, kwargs, result) -> (bytes, tensor-core flops)` or
    `(bytes, tensor-core flops, fp32 flops)`."""

    def __init__(self, table: list[tuple]):
        self.table, self.records, self.saved, self.depth = table, [], [], 0

    def __enter__(self):
        for owner, attr, name, cost in self.table:
            fn = getattr(owner, attr)
            self.saved.append((owner, attr, fn))
            setattr(owner, attr, self._wrap(fn, name, cost))
        return self

    def __exit__(self, *exc):
        for owner, attr, fn in reversed(self.saved):
            setattr(owner, attr, fn)
        self.saved.clear()

    def _wrap(self, fn, name, cost):
        def call(*a, **k):
            if self.depth:
                return fn(*a, **k)
            self.depth += 1
            e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            e0.record()
            out = fn(*a, **k)
            e1.record()
            self.depth -= 1
            label = name(a, out) if callable(name) else name
            self.records.append((label, e0, e1, *cost(a, k, out)))
            return out
        return call

    def summary(self, peaks: dict) -> dict:
        torch.cuda.synchronize()
        acc: dict = {}
        for name, e0, e1, nbytes, flops, *fp32 in self.records:
            r = acc.setdefault(name, [0, 0.0, 0.0])
            floor = max(nbytes / (peaks["hbm_gbs"] * 1e9), flops / (peaks["bf16_tflops"] * 1e12),
                        sum(fp32) / (FP32_TFLOPS * 1e12)) * 1e3
            r[0] += 1
            r[1] += e0.elapsed_time(e1)
            r[2] += floor
        return {n: {"calls": c, "ms": round(ms, 4), "of_roofline": round(fl / ms, 3) if ms else None}
                for n, (c, ms, fl) in sorted(acc.items(), key=lambda kv: -kv[1][1])}


def _linear_cost(a, k, out):
    x, w = a[0], a[1]
    return _bytes(x, w, out), 2.0 * (x.numel() // x.shape[-1]) * w.shape[0] * w.shape[1]


def _linear_name(prefix):
    return lambda a, out: f"{prefix} {a[1].shape[0]}x{a[1].shape[1]}"


def _visited(top: int, experts: int, rows: int) -> float:
    """Expected number of distinct experts of `rows` tokens."""
    return experts * (1.0 - (1.0 - top / experts) ** rows)


def _seen(lengths: list[tuple[int, int]], mask: KeyMask) -> tuple[float, float]:
    """Over (first position, tokens) of a step: key rows its sequences need, and visible (query, key) pairs."""
    keys = pairs = 0
    for start, n in lengths:
        keys += start + n - mask.first(start) + min(mask.keep, mask.first(start))
        for p in range(start, start + n):
            lo = mask.first(p)
            pairs += p + 1 - lo + min(mask.keep, lo)
    return float(keys), float(pairs)


def mezilix_table(z: dict, rows: int, lengths: list[tuple[int, int]]) -> list[tuple]:
    """`lengths`: (first position, tokens) of the step's sequences, `rows` tokens in all."""
    from ..ops import gemm, grouped, latent_attention as latent, moe, stream
    W, H = z["width"], z["heads"]
    keys, pairs = _seen(lengths, KeyMask(z["window"]))
    ew = _visited(z["top"], z["experts"], rows) * z["ff"] * W * 2

    def boundary(a, k, out):
        x, mixer, experts, hist, n = a[0], a[1], a[2], a[3], a[5]
        T = out.shape[0] if isinstance(out, torch.Tensor) else x.shape[0]
        per = 4 + 2 + (0 if experts is None else 2 * experts[2].shape[1]) + 4 * n
        per += 2 if isinstance(out, torch.Tensor) else 4 + 4 + 2 + 2
        return per * T * W, 0.0

    def experts(a, k, out):
        x, w = a[0], a[1]
        return ew + _bytes(x, out), 2.0 * rows * z["top"] * w.shape[1] * w.shape[2]

    return [
        (stream, "embed", "embedding, norm, shift", lambda a, k, o: (a[0].shape[0] * W * (2 + 2 + 4 + 2 + 2), 0.0)),
        (stream, "boundary", "layer boundary", boundary),
        (stream, "final", "final norm", boundary),
        (gemm, "serve_linear", _linear_name("gemm"), _linear_cost),
        (gemm, "matmul_nt", _linear_name("gemm"), _linear_cost),
        (latent, "prepare", "latent norm, rotary, cache write",
         lambda a, k, o: (_bytes(a[0]) * (1 + z["heads"] * z["rot"] / a[0].shape[1]) +
                          a[0].shape[0] * a[1].row_width * 2 * (2 if o is not None else 1), 0.0)),
        (latent, "gather_rows", "latent gather", lambda a, k, o: (2 * _bytes(o), 0.0)),
        (latent, "attend_latent", "attention (latent space)",
         lambda a, k, o: (keys * a[2].row_width * 2 + 2 * _bytes(a[0]), 2.0 * pairs * H * (2 * z["rank"] + z["rot"]))),
        (latent, "attend_expanded", "attention (expanded)",
         lambda a, k, o: (_bytes(a[1], a[2]) + a[0].shape[0] * a[3].q_width * 2 + _bytes(a[7]),
                          2.0 * pairs * H * (z["dim"] + z["rot"] + z["vdim"]))),
        (grouped, "head_linear", lambda a, o: f"per-head projection {a[1].shape[1]}x{a[1].shape[2]}",
         lambda a, k, o: (_bytes(a[0], a[1], o), 2.0 * a[0].shape[0] * a[1].numel())),
        (grouped, "expert_linear", lambda a, o: f"experts {a[1].shape[1]}x{a[1].shape[2]}", experts),
        (moe, "_route_decode", "router top-k, sort", lambda a, k, o: (_bytes(a[0], *o), 0.0)),
        (moe, "_topk_raw", "router top-k", lambda a, k, o: (_bytes(a[0], *o), 0.0)),
        (moe, "make_plan", "routing plan", lambda a, k, o: (_bytes(a[0], o.dest, o.src_of_row), 0.0)),
        (moe, "_permute_raw", "permute", lambda a, k, o: (_bytes(a[0]) + a[1].n * W * 2, 0.0)),
        (moe, "_grouped_act", lambda a, o: f"experts {a[1].shape[1]}x{a[1].shape[2]}",
         lambda a, k, o: (ew + rows * z["top"] * (a[1].shape[1] + a[1].shape[2]) * 2,
                          2.0 * rows * z["top"] * a[1].shape[1] * a[1].shape[2])),
    ]


def vibepel_table(z: dict, rows: int, lengths: list[tuple[int, int]]) -> list[tuple]:
    """The scans' arithmetic is fp32: three products of every state element per token."""
    from ..ops import gemm, grouped, latent_attention as latent, recurrent, stream, window_attention as window
    W, H, G, D = z["width"], z["heads"], z["kv"], z["dim"]
    keys, pairs = _seen(lengths, KeyMask(z["window"]))

    def boundary(a, k, out):
        if isinstance(out, torch.Tensor):                      # last boundary: only the wanted rows
            return out.shape[0] * W * (4 + 2 + 2), 0.0
        return _bytes(*out) + out[0].shape[0] * W * (2 + 4), 0.0

    def state(s, n):                                           # n sequences: S read and written
        return 2 * n * (s.state_width - s.matrix_offset) * 4

    return [
        (stream, "scaled_embed", "embedding", boundary),
        (stream, "postnorm", lambda a, o: "output norm, sum, mixes" if o[1].dim() == 3 else "output norm, sum", boundary),
        (stream, "postnorm_final", "last norms", boundary),
        (gemm, "serve_linear", _linear_name("gemm"), _linear_cost),
        (grouped, "head_linear", lambda a, o: f"gemm 4 x {a[1].shape[1]}x{a[1].shape[2]}",
         lambda a, k, o: (_bytes(a[0], a[1], o), 2.0 * a[0].shape[0] * a[1].numel())),
        (window, "prepare", "head norms, rotary, cache write",
         lambda a, k, o: (a[0].shape[0] * 2 * (2 * (a[1].q_width + a[1].kv_heads * a[1].dim) + a[1].kv_heads * a[1].vdim +
                                               a[1].kv_width), 0.0)),
        (latent, "gather_rows", "key gather", lambda a, k, o: (2 * _bytes(o), 0.0)),
        (window, "attend_rows", "attention (rows)",
         lambda a, k, o: (keys * a[1].kv_width * 2 + a[0].shape[0] * (a[1].q_width + a[1].out_width) * 2, 4.0 * pairs * H * D)),
        (window, "attend_portions", "attention (portions)",
         lambda a, k, o: (a[0].shape[0] * (a[1].q_width + a[1].kv_width + a[1].out_width) * 2, 4.0 * pairs * H * D)),
        (recurrent, "delta_step", "delta rule step",
         lambda a, k, o: (a[0].shape[0] * (a[1].proj_width + a[1].out_width) * 2 + state(a[1], a[0].shape[0]), 0.0)),
        (recurrent, "delta_inputs", "delta rule inputs",
         lambda a, k, o: (a[0].shape[0] * (a[1].channels + 2 * a[1].heads) * 2 + _bytes(*o), 0.0)),
        (recurrent, "delta_scan", "delta rule scan",
         lambda a, k, o: (_bytes(a[0], a[1], o), 0.0, 6.0 * o.numel() * a[2].dim)),
        (recurrent, "gated_norm", "gated norm", lambda a, k, o: (_bytes(a[0]) + 2 * _bytes(a[4]), 0.0)),
        (recurrent, "wkv_step", "WKV step",
         lambda a, k, o: (_bytes(a[0], a[1], a[7]) + state(a[2], a[0].shape[0]), 0.0)),
        (recurrent, "wkv_scan", "WKV scan",
         lambda a, k, o: (_bytes(a[0]) * 3 // 4 + _bytes(a[1], o), 0.0, 6.0 * o.numel() * a[2].dim)),
    ]


def kabulix_table(z: dict, rows: int, lengths: list[tuple[int, int]]) -> list[tuple]:
    from ..ops import gemm, grouped, latent_attention as latent, moe, stream, window_attention as window
    W = z["width"]
    visited = _visited(z["top"], z["experts"], rows)

    def boundary(a, k, out):
        final = isinstance(out, torch.Tensor)                  # last boundary: only the wanted rows
        T = (out if final else out[0]).shape[0]
        per = 4 + 2 + (0 if a[3] is None else 2 * a[3][2].shape[1]) + (0 if final else 4) + 2
        return per * T * W, 0.0

    def kind(s):
        return "chunks" if s.chunked else "window"

    def experts(a, k, out):
        x, w = a[0], a[1]
        cols = out.shape[-1]
        return visited * w.shape[1] * w.shape[2] * 2 + rows * z["top"] * (w.shape[2] + cols) * 2, 2.0 * rows * z["top"] * w.shape[1] * w.shape[2]

    def prepared(a, k, out):
        s = a[1]
        moved = s.q_width + s.kv_heads * s.dim if a[2] is not None else 0       # read and written in place
        return a[0].shape[0] * 2 * (2 * moved + (s.kv_heads * s.vdim if s.values_are_keys else s.kv_width - (moved and s.kv_heads * s.dim)) +
                                    s.kv_width), 0.0

    return [
        (stream, "prenorm_embed", "embedding, norm", lambda a, k, o: (a[0].shape[0] * W * (2 + 4 + 2), 0.0)),
        (stream, "prenorm", lambda a, o: "sum, norm" if a[3] is None else "expert combine, sum, norm", boundary),
        (stream, "prenorm_final", "last norm", boundary),
        (gemm, "serve_linear", _linear_name("gemm"), _linear_cost),
        (gemm, "matmul_nt", _linear_name("gemm"), _linear_cost),
        (window, "prepare", lambda a, o: "bias, head norms, rotary, cache write" if a[2] is not None else "cache write", prepared),
        (latent, "prepare", "latent norm, rotary, cache write",
         lambda a, k, o: (a[0].shape[0] * 2 * (2 * a[1].heads * a[1].rot + a[1].rank + a[1].rot + a[1].row_width * (2 if o is not None else 1)), 0.0)),
        (latent, "gather_rows", "key gather", lambda a, k, o: (2 * _bytes(o), 0.0)),
        (window, "attend_rows", lambda a, o: f"attention ({kind(a[1])}, rows)",
         lambda a, k, o: (_seen(lengths, a[1].mask)[0] * a[1].kv_width * 2 + a[0].shape[0] * (a[1].q_width + a[1].out_width) * 2,
                          2.0 * _seen(lengths, a[1].mask)[1] * a[1].heads * (a[1].dim + a[1].vdim))),
        (window, "attend_portions", lambda a, o: f"attention ({kind(a[1])}, portions)",
         lambda a, k, o: (a[0].shape[0] * (a[1].q_width + a[1].kv_width + a[1].out_width) * 2,
                          2.0 * _seen(lengths, a[1].mask)[1] * a[1].heads * (a[1].dim + a[1].vdim))),
        (latent, "attend_latent", "attention (latent space)",
         lambda a, k, o: (_seen(lengths, a[2].mask)[0] * a[2].row_width * 2 + 2 * _bytes(a[0]),
                          2.0 * _seen(lengths, a[2].mask)[1] * a[2].heads * (2 * a[2].rank + a[2].rot))),
        (latent, "attend_expanded", "attention (latent, portions)",
         lambda a, k, o: (_bytes(a[1], a[2]) + a[0].shape[0] * a[3].q_width * 2 + 2 * _bytes(a[7]),
                          2.0 * _seen(lengths, a[3].mask)[1] * a[3].heads * (a[3].dim + a[3].rot + a[3].vdim))),
        (grouped, "head_linear", lambda a, o: f"per-head projection {a[1].shape[1]}x{a[1].shape[2]}",
         lambda a, k, o: (_bytes(a[0], a[1], o), 2.0 * a[0].shape[0] * a[1].numel())),
        (grouped, "expert_linear", lambda a, o: f"experts {a[1].shape[1]}x{a[1].shape[2]}", experts),
        (moe, "_route_decode", "router top-k, sort", lambda a, k, o: (_bytes(a[0], *o), 0.0)),
        (moe, "_topk_raw", "router top-k", lambda a, k, o: (_bytes(a[0], *o), 0.0)),
        (moe, "make_plan", "routing plan", lambda a, k, o: (_bytes(a[0], o.dest, o.src_of_row), 0.0)),
        (moe, "_permute_raw", "permute", lambda a, k, o: (_bytes(a[0]) + a[1].n * W * 2, 0.0)),
        (moe, "_grouped_act", lambda a, o: f"experts {a[1].shape[1]}x{a[1].shape[2]}", experts),
    ]


def lovurax_table(z: dict, rows: int, lengths: list[tuple[int, int]]) -> list[tuple]:
    from ..ops import gemm, grouped, latent_attention as latent, recurrent, stream, window_attention as window
    W = z["width"]
    keys, pairs = _seen(lengths, KeyMask(UNBOUNDED))

    # key rows per key/value head, and (query, key, head) triples, whose sigmoid weights can count: head norms of ones, scores' addend
    # and temperature of the random model
    from ..models.lovurax import RANDOM_SCORE_ADD
    H, group, longest = z["heads"], z["heads"] // z["kv"], max(start + n for start, n in lengths)
    limit = 1.02 * z["dim"] ** 0.5 * (1.0 + 0.1 * math.log(longest // 4096 + 1))
    seen = [_seen(lengths, KeyMask(window.sigmoid_reach(limit, RANDOM_SCORE_ADD, slope) + 1)) for slope in window.distance_slopes(H).tolist()]
    near_keys = sum(max(k for k, _ in seen[g:g + group]) for g in range(0, H, group)) / z["kv"]
    near_pairs = sum(n for _, n in seen)

    def boundary(a, k, out):
        final = isinstance(out, torch.Tensor)                  # last boundary: only the wanted rows
        T = (out if final else out[0]).shape[0]
        return (4 + 2 + 2 + (0 if final else 4) + 2) * T * W, 0.0

    return [
        (stream, "prenorm_embed", "embedding, norm", lambda a, k, o: (a[0].shape[0] * W * (2 + 4 + 2), 0.0)),
        (stream, "prenorm", "gated sum, norm", boundary),
        (stream, "prenorm_final", "last norm", boundary),
        (gemm, "serve_linear", _linear_name("gemm"), _linear_cost),
        (gemm, "matmul_nt", _linear_name("gemm"), _linear_cost),
        (window, "prepare", "head norms, temperature, cache write",
         lambda a, k, o: (a[0].shape[0] * 2 * (2 * (a[1].q_width + a[1].kv_heads * a[1].dim) + a[1].kv_heads * a[1].vdim +
                                               a[1].kv_width), 0.0)),
        (latent, "prepare", "latent norm, cache write",
         lambda a, k, o: (a[0].shape[0] * 2 * (a[1].rank + a[1].row_width * (2 if o is not None else 1)), 0.0)),
        (latent, "gather_rows", "key gather", lambda a, k, o: (2 * _bytes(o), 0.0)),
        (window, "attend_rows", "attention (sigmoid, rows)",
         lambda a, k, o: (near_keys * a[1].kv_width * 2 + a[0].shape[0] * (a[1].q_width + 2 * a[1].out_width) * 2,
                          2.0 * near_pairs * (a[1].dim + a[1].vdim))),
        (window, "attend_portions", "attention (sigmoid, portions)",
         lambda a, k, o: (a[0].shape[0] * (a[1].q_width + a[1].kv_width + 2 * a[1].out_width) * 2,
                          2.0 * near_pairs * (a[1].dim + a[1].vdim))),
        (latent, "attend_latent", "attention (latent space)",
         lambda a, k, o: (keys * a[2].row_width * 2 + 2 * _bytes(a[0]), 4.0 * pairs * a[2].heads * a[2].rank)),
        (latent, "attend_expanded", "attention (latent, portions)",
         lambda a, k, o: (_bytes(a[1], a[7]) + a[0].shape[0] * a[3].q_width * 2,
                          2.0 * pairs * a[3].heads * (a[3].dim + a[3].vdim))),
        (grouped, "head_linear", lambda a, o: f"per-head projection {a[1].shape[1]}x{a[1].shape[2]}",
         lambda a, k, o: (_bytes(a[0], a[1], o), 2.0 * a[0].shape[0] * a[1].numel())),
        (recurrent, "retention_step", "retention step",
         lambda a, k, o: (a[0].shape[0] * ((a[1].proj_width + a[1].out_width) * 2 + 2 * 4 * a[1].state_width), 0.0)),
        # two fp32 products of every state element per token
        (recurrent, "retention_scan", "retention scan",
         lambda a, k, o: (a[0].shape[0] * (2 * a[1].qk_width + a[1].out_width) * 2 + _bytes(o), 0.0, 4.0 * o.numel() * a[1].dim)),
        (recurrent, "retention_chunks", "retention (chunks, norm, gate)",
         lambda a, k, o: (a[0].shape[0] * (a[1].proj_width + a[1].out_width) * 2, 0.0, 4.0 * a[0].shape[0] * a[1].out_width * a[1].dim)),
        (recurrent, "gated_norm", "gated norm", lambda a, k, o: (_bytes(a[0]) + 2 * _bytes(a[4]), 0.0)),
    ]


def closest_table(z: dict, rows: int, lengths: list[tuple[int, int]], runner) -> list[tuple]:
    from ..ops import activation, gemm, moe, norm, rope
    W, H, D = z["width"], z["heads"], z.get("vdim") or z["dim"]
    keys, pairs = _seen(lengths, KeyMask(UNBOUNDED))
    hkv = z.get("kv") or max(1, H // 4)

    def grouped_cost(a, k, out):
        E, N, K = a[1].shape
        return (_visited(z["top"], E, rows) * N * K * 2 + rows * z["top"] * (N + K) * 2, 2.0 * rows * z["top"] * N * K)

    return [
        (norm, "rmsnorm", "rms norm", lambda a, k, o: (_bytes(a[0], *[t for t in o if t is not None]) + _bytes(*a[3:4]), 0.0)),
        (gemm, "linear", _linear_name("gemm"), _linear_cost),
        (rope, "apply_rope_qkv", "rotary", lambda a, k, o: (2 * _bytes(a[0]) * (H + hkv) / (H + 2 * hkv), 0.0)),
        (runner, "_write_cache", "cache write", lambda a, k, o: (2 * a[1].shape[0] * 2 * hkv * D * 2, 0.0)),
        (runner, "_attend", "attention", lambda a, k, o: (keys * 2 * hkv * D * 2 + 2 * _bytes(o), 4.0 * pairs * H * D)),
        (moe, "topk_softmax", "router top-k", lambda a, k, o: (_bytes(a[0], *o), 0.0)),
        (moe, "make_plan", "routing plan", lambda a, k, o: (_bytes(a[0], o.dest, o.src_of_row), 0.0)),
        (moe, "_permute_raw", "permute", lambda a, k, o: (_bytes(a[0]) + a[1].n * W * 2, 0.0)),
        (moe, "grouped_linear", lambda a, o: f"experts {a[1].shape[1]}x{a[1].shape[2]}", grouped_cost),
        (activation, "glu", "gated activation", lambda a, k, o: (rows * z.get("top", 1) * 3 * o.shape[1] * 2, 0.0)),
        (moe, "_combine_raw", "combine", lambda a, k, o: (rows * z["top"] * W * 2 + _bytes(o), 0.0)),
    ]


# ---------------------------------------------------------------------------------------------- measurement
@dataclass(frozen=True)
class Design:
    sizes: dict
    build: Callable
    closest: Callable
    table: Callable


DESIGNS = {"mezilix": Design(SIZES, build_mezilix, build_closest, mezilix_table),
           "vibepel": Design(VIBEPEL_SIZES, build_vibepel, build_closest_dense, vibepel_table),
           "kabulix": Design(KABULIX_SIZES, build_kabulix, build_closest, kabulix_table),
           "lovurax": Design(LOVURAX_SIZES, build_lovurax, build_closest_dense, lovurax_table)}


def measure(design: str, name: str, peaks: dict, prompts: int = 2, prompt_len: int = 4096, batches=(8, 64), context: int = 2048,
            iters: int = 5) -> dict:
    spec = DESIGNS[design]
    z = spec.sizes[name]
    out: dict = {"sizes": z, "models": {}}
    for kind, build in ((design, spec.build), ("closest", spec.closest)):
        model = build(z)
        core = make_core(model, max(prompts * prompt_len, max(batches) * (context + 64)), max(max(batches), prompts))
        res: dict = {"parameters": sum(p.numel() for p in model.parameters())}

        def table(rows, lengths):
            return spec.table(z, rows, lengths) if kind == design else closest_table(z, rows, lengths, core.runner)

        def profile(step, rows, lengths):
            with OpTimer(table(rows, lengths)) as t:
                torch.cuda._sleep(200_000_000)
                step()
            return t.summary(peaks)

        # prefill: whole prompts in one step
        entries = [StepEntry(i, _tokens(prompt_len, i)) for i in range(prompts)]
        host = HostBatch(core.cache, entries)
        batch = host.to_device("cuda")
        step = lambda: core.runner.forward(batch)   # noqa: E731
        ms = _timed(step, iters)
        T = prompts * prompt_len
        res["prefill"] = {"tokens": T, "ms": ms, "tokens_per_s": T / ms * 1e3,
                          "ops": profile(step, T, [(0, prompt_len)] * prompts)}
        # portions that continue cached prompts
        if kind == design:
            for i in range(prompts):
                core.release(i)
            half = prompt_len // 2
            with torch.no_grad():
                core.execute([StepEntry(i, e.tokens[:half], []) for i, e in enumerate(entries)])
            b2 = HostBatch(core.cache, [StepEntry(i, e.tokens[half:]) for i, e in enumerate(entries)]).to_device("cuda")
            ms = _timed(lambda: core.runner.forward(b2), iters)
            res["prefill_continued"] = {"tokens": T - prompts * half, "ms": ms, "tokens_per_s": (T - prompts * half) / ms * 1e3}
        for i in range(prompts):
            core.release(i)
        # decode: one token per sequence on top of `context` cached tokens
        res["decode"] = {}
        for n in batches:
            for i in range(0, n, 4):
                core.execute([StepEntry(j, _tokens(context, 100 + j), []) for j in range(i, min(n, i + 4))])
            host = HostBatch(core.cache, [StepEntry(j, [j + 1]) for j in range(n)])
            batch = host.to_device("cuda")
            step = lambda: core.runner.logits(core.runner.forward(batch))   # noqa: E731
            d = {"ms": _timed(step, iters), "ops": profile(step, n, [(context, 1)] * n)}
            if core.runner.can_graph(host):
                core.runner.decode_graphed(host)
                d["graph_ms"] = _timed(lambda: core.runner.decode_graphed(host), iters)
            d["tokens_per_s"] = n / min(d["ms"], d.get("graph_ms", math.inf)) * 1e3
            res["decode"][str(n)] = d
            for j in range(n):
                core.release(j)
        out["models"][kind] = res
        del core, model, batch, host, step
        torch.cuda.empty_cache()
    ours, closest = out["models"][design], out["models"]["closest"]
    out[f"{design}_over_closest"] = {
        "prefill": ours["prefill"]["tokens_per_s"] / closest["prefill"]["tokens_per_s"],
        **{f"decode_{n}": ours["decode"][n]["tokens_per_s"] / closest["decode"][n]["tokens_per_s"] for n in ours["decode"]}}
    return out


def run(sizes: list[str], peaks_file: Path, iters: int = 5, design: str = "mezilix") -> dict:
    peaks = {"hbm_gbs": 6538.9, "bf16_tflops": 1608.3}
    try:
        peaks.update(json.loads(peaks_file.read_text()))
    except OSError:
        pass
    from ..ops import _lib
    out = {n: measure(design, n, peaks, iters=iters) for n in sizes}
    _lib.raise_on_loaded_device_error()
    return out
