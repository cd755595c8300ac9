"""Ragged batches: what one step of the engine runs for layer-stack models. Entry e of the batch is a run of tokens that
continues one sequence; prompt portions and single decoded tokens sit side by side in one flat token list. The index
tensors live on the device (csrc/precise.cuh: Ragged), so a decode step over fixed buffers can be captured in a graph."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Optional, Sequence

import torch

TILE = 64       # tokens per tile of the tiled recurrences (csrc/recurrent.cu: LT)


@dataclass
class RaggedBatch:
    tokens: torch.Tensor            # int64 [n]
    cu: torch.Tensor                # int32 [E + 1] first token of every entry
    slot: torch.Tensor              # int32 [E] page-table row and state slot of its sequence
    pos0: torch.Tensor              # int32 [E] position of its first token (< 0: idle slot)
    ent: torch.Tensor               # int32 [n] entry of every token
    lens: Optional[Sequence[int]]   # host copy of the entries' lengths (None: every entry is one token)
    _tiles: Optional[dict] = None

    @property
    def n(self) -> int:
        return self.tokens.shape[0]

    @property
    def entries(self) -> int:
        return self.slot.shape[0]

    @property
    def decode(self) -> bool:
        return self.lens is None

    @classmethod
    def build(cls, work, device) -> "RaggedBatch":
        """`work`: [(slot, position of the first token, token ids)], every entry non-empty."""
        lens = [len(t) for _, _, t in work]
        n, E = sum(lens), len(work)
        ints, cu = [], [0]
        for L in lens:
            cu.append(cu[-1] + L)
        ints = cu + [s for s, _, _ in work] + [p for _, p, _ in work]
        for e, L in enumerate(lens):
            ints += [e] * L
        flat = [int(t) for _, _, toks in work for t in toks]
        meta = torch.tensor(ints, dtype=torch.int32).to(device)
        tokens = torch.tensor(flat, dtype=torch.int64).to(device)
        a, b, c = E + 1, 2 * E + 1, 3 * E + 1
        return cls(tokens, meta[:a], meta[a:b], meta[b:c], meta[c:c + n], None if max(lens) == 1 else lens)

    @classmethod
    def decode_slots(cls, tokens: torch.Tensor, slots: torch.Tensor, positions: torch.Tensor) -> "RaggedBatch":
        """One token per slot over the engine's static buffers (an idle slot has position -1)."""
        B = tokens.shape[0]
        ar = torch.arange(B + 1, dtype=torch.int32, device=tokens.device)
        return cls(tokens, ar, slots, positions, ar[:B], None)

    def tiles(self, size: int = TILE) -> tuple:
        """(first token, entry) of every tile of at most `size` tokens of one entry, the first tile of every entry, and the
        number of tiles. Built once per batch and size: every layer uses the same lists."""
        if self._tiles is None:
            self._tiles = {}
        if size not in self._tiles:
            t0, ent, first, at = [], [], [], 0
            for e, L in enumerate(self.lens if self.lens is not None else [1] * self.entries):
                first.append(len(t0))
                for o in range(0, L, size):
                    t0.append(at + o)
                    ent.append(e)
                at += L
            k = len(t0)
            dev = torch.tensor(t0 + ent + first, dtype=torch.int32).to(self.tokens.device)
            self._tiles[size] = (dev[:k], dev[k:2 * k], dev[2 * k:], k)
        return self._tiles[size]

    def args(self) -> tuple:
        return (self.cu.data_ptr(), self.slot.data_ptr(), self.pos0.data_ptr(), self.ent.data_ptr(), self.entries, self.n)
