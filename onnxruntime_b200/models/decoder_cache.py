"""Cache and state memory of packed decoders: pools of cache blocks and state slots shared by all sequences.

A model declares what it keeps per sequence as a list of ``CacheTensor``: "paged" tensors grow with the sequence and
live in blocks of ``block_size`` tokens named by a block table; "slot" tensors have a fixed size per sequence (recurrent
state) and live in one slot.  ``CachePool`` owns the device tensors and hands blocks and slots to sequences; the graph
updates both in place.  Slots are not cleared between owners: an operator starts from the zero state when a sequence's
past length is 0.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Dict, Hashable, List, Sequence, Tuple

import torch


@dataclass(frozen=True)
class CacheTensor:
    input: str                    # graph input that receives the pool tensor
    output: str                   # graph output bound to the same tensor
    kind: str                     # "paged": [num_blocks, block_size, *shape]; "slot": [num_slots, *shape]
    shape: Tuple[int, ...]
    dtype: torch.dtype


class CacheFull(RuntimeError):
    """No free block or slot is left for a sequence."""


@dataclass
class SequenceEntry:
    slot: int
    blocks: List[int] = field(default_factory=list)
    length: int = 0


class CachePool:
    def __init__(self, spec: Sequence[CacheTensor], num_blocks: int, block_size: int, num_slots: int, device: torch.device):
        self.spec = list(spec)
        self.num_blocks, self.block_size, self.num_slots = num_blocks, block_size, num_slots
        # zero-filled once: attention kernels read whole tiles and multiply what lies beyond a sequence's end by zero, so
        # every entry has to be finite
        self.tensors = {c.input: torch.zeros((num_blocks, block_size, *c.shape) if c.kind == "paged" else (num_slots, *c.shape),
                                             dtype=c.dtype, device=device) for c in self.spec}
        self.free_blocks = list(range(num_blocks - 1, -1, -1))   # popped from the end: block 0 first, freed blocks first
        self.free_slots = list(range(num_slots - 1, -1, -1))
        self.sequences: Dict[Hashable, SequenceEntry] = {}

    def open(self, seq: Hashable) -> SequenceEntry:
        if seq in self.sequences:
            raise ValueError(f"sequence {seq!r} is already open")
        if not self.free_slots:
            raise CacheFull(f"all {self.num_slots} sequence slots are in use")
        entry = SequenceEntry(self.free_slots.pop())
        self.sequences[seq] = entry
        return entry

    def reserve(self, seq: Hashable, tokens: int) -> bool:
        """Room for ``tokens`` more tokens of ``seq``; True when blocks were added.  All or nothing."""
        entry = self.sequences[seq]
        need = (entry.length + tokens + self.block_size - 1) // self.block_size - len(entry.blocks)
        if need > len(self.free_blocks):
            raise CacheFull(f"sequence {seq!r} needs {need} more cache blocks, {len(self.free_blocks)} are free")
        for _ in range(max(need, 0)):
            entry.blocks.append(self.free_blocks.pop())
        return need > 0

    def advance(self, seq: Hashable, tokens: int) -> None:
        self.sequences[seq].length += tokens

    def close(self, seq: Hashable) -> None:
        entry = self.sequences.pop(seq)
        self.free_blocks.extend(reversed(entry.blocks))
        self.free_slots.append(entry.slot)

    def copy_sequence_state(self, sources: Sequence[Hashable], targets: Sequence[Hashable]) -> None:
        """Content of ``targets[i]`` becomes that of ``sources[i]`` (beam search); all open, with equally many blocks."""
        src, dst = [self.sequences[s] for s in sources], [self.sequences[t] for t in targets]
        src_blocks = [b for e in src for b in e.blocks]
        dst_blocks = [b for e in dst for b in e.blocks]
        if any(len(a.blocks) != len(b.blocks) for a, b in zip(src, dst)):
            raise ValueError("sequences hold different numbers of blocks")
        lengths = [e.length for e in src]
        for c in self.spec:
            t = self.tensors[c.input]
            a = torch.tensor(src_blocks if c.kind == "paged" else [e.slot for e in src], device=t.device)
            b = torch.tensor(dst_blocks if c.kind == "paged" else [e.slot for e in dst], device=t.device)
            t.index_copy_(0, b, t.index_select(0, a))
        for e, n in zip(dst, lengths):
            e.length = n
