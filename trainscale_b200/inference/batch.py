"""One engine step as a flattened token batch: which sequence brings which tokens, and everything on the device that the
layers need to find its keys, its state and the rows whose logits are wanted."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ..ops.masks import KeyMask
from ..ops.stream import ROW_BEFORE
from .kv_cache import PagedKVCache


@dataclass
class StepEntry:
    """A request's next tokens.  `want`: places among them whose logits are asked for (None: the last one)."""
    seq_id: int
    tokens: list[int]
    want: list[int] | None = None
    adapter: int = 0              # LoRA adapter index (engines with adapters loaded)

    @property
    def wanted(self) -> list[int]:
        return [len(self.tokens) - 1] if self.want is None else self.want


@dataclass
class PromptContext:
    """Keys of the batch's multi-token entries for one mask: the sequences' rows in key order."""
    cu_q: torch.Tensor            # int32 [n + 1], query rows (relative to the first multi-token row)
    cu_k: torch.Tensor            # int32 [n + 1], key rows
    max_q: int
    slots: torch.Tensor | None    # cache slot of every key row; None: the keys are exactly the new tokens


@dataclass
class Portions:
    """The batch's multi-token entries, by row relative to the first multi-token row."""
    offsets: list[int]            # [count + 1]
    cu: torch.Tensor              # int32 copy on the device

    @property
    def count(self) -> int:
        return len(self.offsets) - 1

    @property
    def longest(self) -> int:
        return max(b - a for a, b in zip(self.offsets[:-1], self.offsets[1:]))


class HostBatch:
    """Host side of a step: tokens are appended to the cache, index lists are built.  Single-token entries come first
    (`order` maps batch position -> entry), so that decoding rows and portions of prompts are contiguous."""

    def __init__(self, cache: PagedKVCache, entries: list[StepEntry]):
        self.cache = cache
        self.order = sorted(range(len(entries)), key=lambda i: len(entries[i].tokens) > 1)
        self.seq_ids, self.q_lens, self.starts = [], [], []
        self.tok, self.prev, self.pos, self.slots = [], [], [], []
        self.row_seq, self.row_prev, self.row_next, self.adapters = [], [], [], []
        self.out_rows: list[int] = []
        self.out_entry: list[int] = []      # entry of every output row
        for b, i in enumerate(self.order):
            e = entries[i]
            n, row0 = len(e.tokens), len(self.tok)
            x = cache.extend(e.seq_id, e.tokens)
            self.seq_ids.append(e.seq_id)
            self.q_lens.append(n)
            self.starts.append(x.start)
            self.tok += e.tokens
            self.prev += [x.prev_token] + e.tokens[:-1]
            self.pos += range(x.start, x.start + n)
            self.slots += x.slots
            self.row_seq += [b] * n
            self.row_prev += [x.state_read] + [ROW_BEFORE] * (n - 1)
            self.row_next += [-1] * (n - 1) + [x.state_write]
            self.adapters += [e.adapter] * n
            self.out_rows += [row0 + w for w in e.wanted]
            self.out_entry += [i] * len(e.wanted)
        self.n_single = sum(n == 1 for n in self.q_lens)

    @property
    def all_single(self) -> bool:
        return self.n_single == len(self.q_lens)

    def to_device(self, device, with_adapters: bool = False) -> "StepBatch":
        bt, sl = self.cache.block_table(self.seq_ids, None)
        parts32 = [self.prev, self.pos, self.row_seq, self.row_prev, self.row_next, self.out_rows]
        i32 = torch.tensor([v for p in parts32 for v in p], dtype=torch.int32)
        i64 = torch.tensor(self.tok + self.slots + (self.adapters if with_adapters else []), dtype=torch.int64)
        # three copies for the whole step
        i32 = torch.cat([i32, bt.reshape(-1), sl]).to(device)
        i64 = i64.to(device)
        views, at = [], 0
        for n in [len(p) for p in parts32] + [bt.numel(), sl.numel()]:
            views.append(i32[at:at + n])
            at += n
        prev, pos, row_seq, row_prev, row_next, out_rows, table, lens = views
        T = len(self.tok)
        return StepBatch(self, i64[:T], prev, pos, i64[T:2 * T], table.view(bt.shape), lens, row_seq, row_prev, row_next,
                         out_rows, self.n_single, max(int(sl.max()), 1), all(s == 0 for s in self.starts),
                         i64[2 * T:] if with_adapters else None)


@dataclass
class StepBatch:
    host: HostBatch | None            # None: static buffers of a captured decode step
    token_ids: torch.Tensor           # int64 [T]
    prev_tokens: torch.Tensor         # int32 [T], -1 for a sequence's first token
    positions: torch.Tensor           # int32 [T]
    slots: torch.Tensor               # int64 [T]
    block_table: torch.Tensor         # int32 [sequences, blocks]
    seq_lens: torch.Tensor            # int32 [sequences], after this step's tokens
    row_seq: torch.Tensor             # int32 [T]
    row_prev: torch.Tensor            # int32 [T] (ops/stream.StreamRows)
    row_next: torch.Tensor            # int32 [T]
    out_rows: torch.Tensor            # int32: rows whose logits are wanted
    n_single: int                     # leading rows that are single-token entries
    max_len: int                      # upper bound of seq_lens
    fresh: bool                       # every sequence starts at position 0
    adapter_ids: torch.Tensor | None = None
    splits: int | None = None         # captured decode: split count of the block-table width
    _contexts: dict = field(default_factory=dict)

    @property
    def captured(self) -> bool:
        """A decode step that is (being) recorded as a CUDA graph over static buffers."""
        return self.host is None

    @property
    def num_tokens(self) -> int:
        return self.token_ids.shape[0]

    @property
    def seq_ids(self) -> list[int]:
        return self.host.seq_ids

    @property
    def q_lens(self) -> list[int]:
        return self.host.q_lens if self.host is not None else [1] * self.num_tokens

    @property
    def cu_q(self) -> torch.Tensor:
        """int32 [sequences + 1]: first row of every sequence (uploaded once per step)."""
        if "cu_q" not in self._contexts:
            cu = [0]
            for n in self.q_lens:
                cu.append(cu[-1] + n)
            self._contexts["cu_q"] = torch.tensor(cu, dtype=torch.int32).to(self.token_ids.device)
        return self._contexts["cu_q"]

    @property
    def portions(self) -> Portions | None:
        """Row offsets of the multi-token entries (None: no such entries)."""
        if self.host is None or self.host.all_single:
            return None
        if "portions" not in self._contexts:
            at = [0]
            for n in self.host.q_lens[self.host.n_single:]:
                at.append(at[-1] + n)
            self._contexts["portions"] = Portions(at, torch.tensor(at, dtype=torch.int32).to(self.token_ids.device))
        return self._contexts["portions"]

    def prompt_context(self, mask: KeyMask) -> PromptContext | None:
        """Key rows that the multi-token entries see through `mask` (None: no such entries)."""
        if self.host is None or self.host.all_single:
            return None
        if mask not in self._contexts:
            h = self.host
            first = h.n_single          # entries and rows before it are single tokens
            cu_q, cu_k, slots = [0], [0], []
            fresh = all(s == 0 for s in h.starts[first:])
            bs = h.cache.block_size
            for sid, start, n in zip(h.seq_ids[first:], h.starts[first:], h.q_lens[first:]):
                lo = mask.first(start)
                kept = min(mask.keep, lo)
                cu_q.append(cu_q[-1] + n)
                cu_k.append(cu_k[-1] + kept + start + n - lo)
                if not fresh:
                    j = torch.cat([torch.arange(kept), torch.arange(lo, start + n)])
                    slots.append(torch.tensor(h.cache.seqs[sid].blocks)[j // bs] * bs + j % bs)
            dev = self.token_ids.device
            cu = torch.tensor(cu_q + cu_k, dtype=torch.int32).to(dev)
            self._contexts[mask] = PromptContext(cu[:len(cu_q)], cu[len(cu_q):], max(h.q_lens[first:]),
                                                 None if fresh else torch.cat(slots).to(dev))
        return self._contexts[mask]
