"""Bookkeeping of live sequences: cache blocks, state slots and lengths.  Host side only — the device buffers that blocks
and slots index belong to the model (`LlamaDecoder`'s paged KV cache, `HybridState`)."""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Optional


class OutOfCache(RuntimeError):
    """No free cache block or state slot: the caller waits for a sequence to end, or refuses the request."""


NO_BLOCK = -1


@dataclass
class Sequence:
    """One live sequence: its state slot, its cache blocks in order of position (NO_BLOCK where the window has passed), and how
    many tokens they stand for."""
    name: Hashable
    slot: int
    blocks: List[int] = field(default_factory=list)
    length: int = 0
    passed: int = 0                  # blocks before this one have been looked at by `SequenceTable.advance`

    @property
    def held(self) -> int:
        return sum(b != NO_BLOCK for b in self.blocks)


class SequenceTable:
    """Hands out `num_blocks` cache blocks of `block_size` tokens and `max_sequences` state slots.  What a sequence held is
    free for the next one as soon as it is closed.

    `window`, `keep_first`: every layer's attention sees the last `window` tokens and the first `keep_first` only (the largest of
    each over the layers).  Blocks that no later token sees are handed back while the sequence runs."""

    def __init__(self, num_blocks: int, block_size: int, max_sequences: int, window: Optional[int] = None, keep_first: int = 0):
        if num_blocks < 1 or block_size < 1 or max_sequences < 1:
            raise ValueError("a sequence table needs at least one block, one token per block and one slot")
        if window is not None and (window < 1 or keep_first < 0):
            raise ValueError("a window holds at least the token itself")
        self.window, self.keep_first = window, keep_first
        self.num_blocks, self.block_size, self.max_sequences = num_blocks, block_size, max_sequences
        self._free_blocks = list(range(num_blocks - 1, -1, -1))
        self._free_slots = list(range(max_sequences - 1, -1, -1))
        self.live: Dict[Hashable, Sequence] = {}

    @property
    def free_blocks(self) -> int:
        return len(self._free_blocks)

    @property
    def free_slots(self) -> int:
        return len(self._free_slots)

    def open(self, name: Hashable) -> Sequence:
        if name in self.live:
            raise ValueError(f"sequence {name!r} is already open")
        if not self._free_slots:
            raise OutOfCache("no free state slot")
        seq = Sequence(name, self._free_slots.pop())
        self.live[name] = seq
        return seq

    def blocks_needed(self, seq: Sequence, tokens: int) -> int:
        return max(0, -(-(seq.length + tokens) // self.block_size) - len(seq.blocks))

    def extend(self, seq: Sequence, tokens: int) -> None:
        """Room for `tokens` more tokens (all or nothing); `advance` counts them once they have run."""
        need = self.blocks_needed(seq, tokens)
        if need > len(self._free_blocks):
            raise OutOfCache(f"{need} cache blocks needed, {len(self._free_blocks)} free")
        for _ in range(need):
            seq.blocks.append(self._free_blocks.pop())

    def advance(self, seq: Sequence, tokens: int) -> None:
        seq.length += tokens
        if self.window is None:
            return
        kept = -(-self.keep_first // self.block_size)
        unseen = max(0, seq.length - self.window + 1) // self.block_size          # whole blocks before the next token's window
        for i in range(max(seq.passed, kept), unseen):
            self._free_blocks.append(seq.blocks[i])
            seq.blocks[i] = NO_BLOCK
        seq.passed = max(seq.passed, unseen)

    def most_blocks(self, tokens: int, portion: int) -> int:
        """The most blocks that a sequence of `tokens` tokens, fed at most `portion` at a time, ever holds."""
        whole = -(-tokens // self.block_size)
        if self.window is None:
            return whole
        return min(whole, -(-self.keep_first // self.block_size) + -(-(self.window - 1 + portion) // self.block_size) + 1)

    def close(self, name: Hashable) -> None:
        seq = self.live.pop(name)
        self._free_blocks.extend(b for b in reversed(seq.blocks) if b != NO_BLOCK)
        self._free_slots.append(seq.slot)
