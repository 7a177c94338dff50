"""What decoders with their own serving path have in common: parameters, checkpoints, whole-sequence logits, construction.

A subclass sets `config`, `embed` and `layers` (modules with a `mixer`), names its stored tensors in `_checkpoint_tensors`, and
defines `cache_spec`, `serve` and `logits` for the engine."""
from __future__ import annotations

import torch
import torch.nn as nn


def fp32_param(*shape) -> nn.Parameter:
    return nn.Parameter(torch.empty(*shape, dtype=torch.float32), requires_grad=False)


def weight_param(*shape) -> nn.Parameter:
    return nn.Parameter(torch.zeros(*shape), requires_grad=False)     # padding rows and columns stay zero


def up8(n: int) -> int:
    return -(-n // 8) * 8


def require(ok: bool, layer: int, what: str) -> None:
    if not ok:
        raise ValueError(f"layer {layer}: needs {what}")


class ServedDecoder(nn.Module):
    # libraries `serve` needs (compiled together at the first use)
    LIBRARIES: tuple[str, ...] = ()

    def __init__(self):
        super().__init__()
        self._side = None                 # second stream of captured decode steps

    # ---------------------------------------------------------------- weights
    def _checkpoint_tensors(self):
        """(checkpoint name, parameter, view or packed part of one) of every stored tensor."""
        raise NotImplementedError

    def finalize(self) -> None:
        """What is derived from the weights, after they changed."""

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
        self.finalize()

    @torch.no_grad()
    def to_checkpoint(self) -> dict[str, torch.Tensor]:
        return {name: t.detach().to(torch.bfloat16).contiguous() for name, t in self._checkpoint_tensors()}

    # ---------------------------------------------------------------- serving
    def _side_stream(self) -> "torch.cuda.Stream":
        if self._side is None:
            self._side = torch.cuda.Stream(device=self.embed.device)
        return self._side

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

    # ---------------------------------------------------------------- construction
    @classmethod
    def empty(cls, config, dtype, device) -> "ServedDecoder":
        device = torch.device(device or "cpu")
        if device.type == "cuda":
            from ..ops import _lib
            _lib.prepare(list(cls.LIBRARIES))
        prev = torch.get_default_dtype()
        torch.set_default_dtype(dtype)
        try:
            with torch.device(device):
                return cls(config).eval()
        finally:
            torch.set_default_dtype(prev)

    @classmethod
    def random(cls, config, dtype, device, seed: int | None) -> "ServedDecoder":
        model = cls.empty(config, dtype, device)
        model.reset_parameters(0 if seed is None else seed)
        return model

    @classmethod
    def from_checkpoint(cls, config, state_dict: dict[str, torch.Tensor], dtype, device) -> "ServedDecoder":
        model = cls.empty(config, dtype, device)
        model.load_checkpoint(state_dict)
        return model
