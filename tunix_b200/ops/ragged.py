"""Ragged batches: what one step of the engine runs for layer-stack models. Entry e of the batch is a run of tokens that
continues one sequence; prompt portions and single decoded tokens sit side by side in one flat token list. The index
tensors live on the device (csrc/precise.cuh: Ragged), so a decode step over fixed buffers can be captured in a graph."""
from __future__ import annotations

from dataclasses import dataclass
from typing import NamedTuple, Optional, Sequence

import numpy as np
import torch

TILE = 64       # tokens per tile of the tiled recurrences (csrc/recurrent.cu: LT)
EXPAND_MIN, EXPAND_RATIO = 16, 8    # shortest portion whose keys are expanded from latents, and most cached rows per token of it


class LatentPlan(NamedTuple):
    """How a batch attends to cached latents. Portions of prompts read keys and values that are expanded for the call, in blocks of
    64 positions; the other entries' tokens attend in the absorbed form, one by one."""
    blocks: Optional[tuple]         # int32 (page-table row, first position) of every block to expand; None: no such portion
    table: Optional[torch.Tensor]   # int32 [entries, ..]: block of every 64 positions of an entry, as a page table
    tiles: Optional[tuple]          # query tiles of those portions: (first token, entry, number)
    entries: Optional[torch.Tensor]     # int32 0 .. entries - 1: the table's rows
    rows: Optional[torch.Tensor]    # int32: the tokens of the other entries; None: every token of the batch
    slots: Optional[torch.Tensor]   # their page-table rows
    lens: Optional[torch.Tensor]    # and the keys each sees at most


@dataclass
class RaggedBatch:
    tokens: torch.Tensor            # int64 [n]
    cu: torch.Tensor                # int32 [E + 1] first token of every entry
    slot: torch.Tensor              # int32 [E] page-table row and state slot of its sequence
    pos0: torch.Tensor              # int32 [E] position of its first token (< 0: idle slot)
    ent: torch.Tensor               # int32 [n] entry of every token
    lens: Optional[Sequence[int]]   # host copy of the entries' lengths (None: every entry is one token)
    work: Optional[list] = None     # host copy of (slot, position of the first token) of every entry
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
        return cls(tokens, meta[:a], meta[a:b], meta[b:c], meta[c:c + n], None if max(lens) == 1 else lens, [w[:2] for w in work])

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

    def latent_plan(self, window: int) -> LatentPlan:
        """Built once per batch and window. A portion is expanded when it is long enough to pay for the window before it."""
        if self.lens is None:
            return LatentPlan(None, None, None, None, None, self.slot, None)
        if self._tiles is None:
            self._tiles = {}
        key = ("latent", window)
        if key not in self._tiles:
            b_slot, b_pos, t0, t_ent, spans, rows, slots, lens, at = [], [], [], [], [], [], [], [], 0
            for e, (L, (slot, p0)) in enumerate(zip(self.lens, self.work)):
                before = min(p0, window - 1) if window > 0 else p0
                if L >= EXPAND_MIN and L * EXPAND_RATIO >= before:
                    first = (p0 - before) // 64
                    count = -(-(p0 + L) // 64) - first
                    spans.append((e, first, len(b_pos), count))
                    b_slot += [slot] * count
                    b_pos += range(first * 64, (first + count) * 64, 64)
                    t0 += range(at, at + L, 128)
                    t_ent += [e] * (-(-L // 128))
                else:
                    rows += range(at, at + L)
                    slots += [slot] * L
                    lens += range(p0 + 1, p0 + L + 1)
                at += L
            table = np.zeros((len(self.lens), max((f + c for _, f, _, c in spans), default=1)), np.int32)
            for e, f, b, c in spans:
                table[e, f:f + c] = np.arange(b, b + c)
            E, nb, nt, nr = len(self.lens), len(b_pos), len(t0), len(rows)
            flat = np.concatenate([np.asarray(x, np.int32) for x in (table.ravel(), b_slot, b_pos, t0, t_ent, range(E), rows, slots, lens)])
            parts = torch.from_numpy(flat).to(self.tokens.device).split([table.size, nb, nb, nt, nt, E, nr, nr, nr])
            self._tiles[key] = LatentPlan((parts[1], parts[2]) if nb else None, parts[0].view(E, -1), (parts[3], parts[4], nt), parts[5],
                                          parts[6], parts[7], parts[8])
        return self._tiles[key]

    def args(self) -> tuple:
        return (self.cu.data_ptr(), self.slot.data_ptr(), self.pos0.data_ptr(), self.ent.data_ptr(), self.entries, self.n)
