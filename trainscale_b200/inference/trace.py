"""Trace replay: given token ids go through the engine step by step, and the logits that are asked for are written out.

Nothing is sampled.  Every input line is one engine step (`EngineCore.execute`): the model, cache, state slots, kernels and
captured decode graphs are those of generation; only the scheduler's choice of tokens is replaced by the trace.

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

`entries` is one batch; `want` are places among an entry's tokens; requests named in `end` give back what they hold after
the step.  Wanted logits go to <out>/<step>.f32 (little-endian float32 [wanted, vocab]); `done <step>` follows on stdout.
"""
from __future__ import annotations

import argparse
import json
import sys
from pathlib import Path

import torch

from .engine import EngineConfig, EngineCore
from .batch import StepEntry

MAX_REQUESTS = 4


class TraceRunner:
    def __init__(self, core: EngineCore):
        self.core = core
        self.ids: dict[str, int] = {}         # live requests -> cache sequence
        self._next = 0

    def run(self, record: dict) -> torch.Tensor | None:
        """One step; the wanted logits [wanted, vocab] or None."""
        entries = []
        for e in record["entries"]:
            if e["id"] not in self.ids:
                self.ids[e["id"]] = self._next
                self._next += 1
            entries.append(StepEntry(self.ids[e["id"]], list(e["tokens"]), list(e.get("want") or [])))
        logits = self.core.execute(entries) if entries else None
        for name in record.get("end") or []:
            self.core.release(self.ids.pop(name))
        if not any(e.want for e in entries):
            return None
        return logits


def build_core(model: str, dtype: str, max_tokens: int, device: str = "cuda") -> EngineCore:
    cfg = EngineConfig(model=model, dtype=dtype, device=device, enforce_eager=False)
    cfg.scheduler.max_num_seqs = MAX_REQUESTS
    cfg.cache.num_gpu_blocks = -(-max_tokens // cfg.cache.block_size)
    cfg.cache.max_model_len = max_tokens
    return EngineCore(cfg)


def main(argv: list[str] | None = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens the cache holds for all live requests together")
    a = ap.parse_args(argv)
    if not torch.cuda.is_available():
        print("trace_run needs a CUDA device", file=sys.stderr)
        return 1
    torch.set_float32_matmul_precision("highest")      # float32 means float32: no TF32 products
    from ..ops import _lib
    runner = TraceRunner(build_core(a.model, a.dtype, a.max_tokens))
    out = Path(a.out)
    for line in sys.stdin:
        if not line.strip():
            continue
        record = json.loads(line)
        logits = runner.run(record)
        if logits is not None:
            logits.float().cpu().numpy().astype("<f4").tofile(out / f"{record['step']}.f32")
        print(f"done {record['step']}", flush=True)
    _lib.raise_on_loaded_device_error()
    return 0


if __name__ == "__main__":
    sys.exit(main())
