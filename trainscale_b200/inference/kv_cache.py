"""Paged cache: fixed-size blocks, per-sequence block tables, prefix sharing by reference counts, and state slots for
models that carry something per sequence from step to step besides the paged entries."""
from __future__ import annotations

import hashlib
import math
from dataclasses import dataclass, field

import torch


class BlockAllocator:
    """Reference-counted blocks. A released block whose content is indexed by a prefix hash stays reusable (it moves
    to an LRU pool and is only overwritten when no plain free block is left)."""

    def __init__(self, num_blocks: int):
        from collections import OrderedDict
        self.num_blocks = num_blocks
        self.free = list(range(num_blocks - 1, -1, -1))
        self.free_cached: "OrderedDict[int, None]" = OrderedDict()
        self.ref = [0] * num_blocks
        self.prefix_index: dict[bytes, int] = {}     # hash of a full block's tokens (+ parent hash) -> block id
        self.block_hash: dict[int, bytes] = {}

    @property
    def num_free(self) -> int:
        return len(self.free) + len(self.free_cached)

    def allocate(self) -> int:
        if self.free:
            b = self.free.pop()
        elif self.free_cached:
            b, _ = self.free_cached.popitem(last=False)      # evict the least recently released cached block
            h = self.block_hash.pop(b, None)
            if h is not None and self.prefix_index.get(h) == b:
                del self.prefix_index[h]
        else:
            raise MemoryError("KV cache is out of blocks")
        self.ref[b] = 1
        return b

    def share(self, b: int) -> int:
        if self.ref[b] == 0:
            self.free_cached.pop(b, None)
        self.ref[b] += 1
        return b

    def release(self, b: int) -> None:
        self.ref[b] -= 1
        if self.ref[b] == 0:
            if b in self.block_hash:
                self.free_cached[b] = None
            else:
                self.free.append(b)


@dataclass
class CacheSpec:
    """What a model keeps per token and per sequence.

    `paged`: for every layer, name -> shape of one token's entry (in the cache dtype), e.g. {"k": (Hkv, D), "v": (Hkv, D)}
    or {"latent": (width,)}.  `state`: for every layer, the width of the sequence's fp32 state row (0: none)."""
    paged: list[dict[str, tuple[int, ...]]]
    state: list[int] = field(default_factory=list)

    @classmethod
    def kv(cls, num_layers: int, n_kv_heads: int, head_dim: int) -> "CacheSpec":
        return cls([{"k": (n_kv_heads, head_dim), "v": (n_kv_heads, head_dim)} for _ in range(num_layers)])

    @property
    def has_state(self) -> bool:
        return any(self.state)

    def bytes_per_token(self, element_size: int) -> int:
        return sum(element_size * math.prod(shape) for layer in self.paged for shape in layer.values())

    def bytes_per_sequence(self) -> int:
        return 2 * 4 * sum(self.state)


@dataclass
class SequenceBlocks:
    blocks: list[int] = field(default_factory=list)
    num_tokens: int = 0
    last_token: int = -1          # token at num_tokens - 1 (-1: none yet)
    slot: int = -1                # state slot (-1: none held)
    phase: int = 0                # which of the slot's two rows holds the current state


@dataclass
class Extension:
    """One sequence's share of a step: where its new tokens go and what they continue from."""
    start: int                    # position of the first new token
    slots: list[int]              # flat cache slot of every new token
    prev_token: int               # token before the first new one (-1: none)
    state_read: int               # state row left by the step before (-1: none, or the model has no state)
    state_write: int              # state row this step leaves (-1: the model has no state)


class PagedKVCache:
    """Paged entries [layers][num_blocks, block_size, ...] and state rows [layers][2 * slots + 1, width].

    The default spec is keys and values per head (`k`, `v`); `spec` describes any other layout (`entries[layer][name]`).
    A sequence with state owns a slot of TWO rows: a step reads one and writes the other, so that rows of one launch
    never overwrite what other rows of it still read.  A model with state cannot take up a sequence in the middle of
    a shared prefix (the state there is not kept), so prefix sharing is off for it."""

    def __init__(self, num_layers: int, num_blocks: int, block_size: int, n_kv_heads: int = 0, head_dim: int = 0, dtype=None,
                 device=None, enable_prefix_caching: bool = True, spec: CacheSpec | None = None, state_slots: int = 0):
        self.block_size, self.num_layers = block_size, num_layers
        self.spec = spec or CacheSpec.kv(num_layers, n_kv_heads, head_dim)
        self.alloc = BlockAllocator(num_blocks)
        # one block beyond the allocator's range: padding rows of a fixed-shape (CUDA-graph) decode batch write their
        # entries there and read them back as their one-token "sequence"; their state goes to the spare row
        self.trash_block = num_blocks
        self.entries = [{name: torch.zeros((num_blocks + 1, block_size, *shape), dtype=dtype, device=device)
                         for name, shape in layer.items()} for layer in self.spec.paged]
        self.k = [e.get("k") for e in self.entries]
        self.v = [e.get("v") for e in self.entries]
        self.state_slots = state_slots if self.spec.has_state else 0
        self.trash_state = 2 * self.state_slots
        self.state = [torch.zeros(2 * self.state_slots + 1, w, dtype=torch.float32, device=device) if w else None
                      for w in self.spec.state]
        self.free_slots = list(range(self.state_slots - 1, -1, -1))
        self.seqs: dict[int, SequenceBlocks] = {}
        self.prefix_caching = enable_prefix_caching and not self.spec.has_state
        self.prefix_hits = 0

    def blocks_needed(self, seq_id: int, new_tokens: int) -> int:
        s = self.seqs.get(seq_id)
        have = len(s.blocks) * self.block_size if s else 0
        used = s.num_tokens if s else 0
        return max(0, -(-(used + new_tokens - have) // self.block_size))

    def can_append(self, seq_id: int, new_tokens: int) -> bool:
        return self.blocks_needed(seq_id, new_tokens) <= self.alloc.num_free

    def match_prefix(self, seq_id: int, tokens: list[int], salt: bytes = b"") -> int:
        """Reuse cached full blocks that hold the same token prefix; returns the number of tokens covered.
        `salt` separates caches whose keys / values differ for the same tokens (e.g. another LoRA adapter)."""
        s = self.seqs.setdefault(seq_id, SequenceBlocks())
        if not self.prefix_caching or s.blocks:
            return 0
        parent = salt
        covered = 0
        # never cover the whole prompt: at least one token must run through the model to produce logits
        for i in range(0, max(0, len(tokens) - 1) // self.block_size * self.block_size, self.block_size):
            h = hashlib.sha1(parent + str(tokens[i:i + self.block_size]).encode()).digest()
            b = self.alloc.prefix_index.get(h)
            if b is None:
                break
            s.blocks.append(self.alloc.share(b))
            covered += self.block_size
            parent = h
        s.num_tokens = covered
        if covered:
            s.last_token = tokens[covered - 1]
            self.prefix_hits += covered
        return covered

    def append_slots(self, seq_id: int, n: int) -> list[int]:
        """Reserve n token slots at the end of the sequence; returns flat slot ids (block * block_size + offset)."""
        s = self.seqs.setdefault(seq_id, SequenceBlocks())
        slots = []
        for _ in range(n):
            if s.num_tokens == len(s.blocks) * self.block_size:
                s.blocks.append(self.alloc.allocate())
            b = s.blocks[s.num_tokens // self.block_size]
            slots.append(b * self.block_size + s.num_tokens % self.block_size)
            s.num_tokens += 1
        return slots

    def extend(self, seq_id: int, tokens: list[int]) -> Extension:
        """Make room for `tokens` at the end of the sequence (created at its first call)."""
        s = self.seqs.setdefault(seq_id, SequenceBlocks())
        read = write = -1
        if self.spec.has_state:
            if s.slot < 0:
                if not self.free_slots:
                    raise MemoryError("every state slot is in use")
                s.slot = self.free_slots.pop()
            if s.num_tokens:
                read = 2 * s.slot + s.phase
            s.phase ^= 1
            write = 2 * s.slot + s.phase
        start, prev = s.num_tokens, s.last_token
        slots = self.append_slots(seq_id, len(tokens))
        s.last_token = tokens[-1]
        return Extension(start, slots, prev, read, write)

    def register_full_blocks(self, seq_id: int, tokens: list[int], salt: bytes = b"") -> None:
        if not self.prefix_caching:
            return
        s = self.seqs[seq_id]
        parent = salt
        # (a token that was sampled last has not been through the model: its entry is not in the cache yet)
        for bi in range(min(len(s.blocks), min(len(tokens), s.num_tokens) // self.block_size)):
            h = hashlib.sha1(parent + str(tokens[bi * self.block_size:(bi + 1) * self.block_size]).encode()).digest()
            b = s.blocks[bi]
            if h not in self.alloc.prefix_index:
                self.alloc.prefix_index[h] = b
                self.alloc.block_hash[b] = h
            parent = h

    def free_sequence(self, seq_id: int) -> None:
        s = self.seqs.pop(seq_id, None)
        if s:
            for b in s.blocks:
                self.alloc.release(b)
            if s.slot >= 0:
                self.free_slots.append(s.slot)

    def block_table(self, seq_ids: list[int], device) -> tuple[torch.Tensor, torch.Tensor]:
        mx = max((len(self.seqs[i].blocks) for i in seq_ids), default=1)
        bt = torch.zeros(len(seq_ids), max(mx, 1), dtype=torch.int32)
        for r, i in enumerate(seq_ids):
            b = self.seqs[i].blocks
            bt[r, :len(b)] = torch.tensor(b, dtype=torch.int32)
        lens = torch.tensor([self.seqs[i].num_tokens for i in seq_ids], dtype=torch.int32)
        if device is None:
            return bt, lens
        return bt.to(device), lens.to(device)

    def utilization(self) -> float:
        return 1.0 - self.alloc.num_free / self.alloc.num_blocks
