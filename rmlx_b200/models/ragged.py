"""Ragged batches: one forward pass over the new tokens of several sequences at once, prompt portions
beside single decoded tokens.

``RaggedBatch`` turns (sequence, tokens) entries into the device arrays the kernels read: token ids,
positions, the block-table row of every token, the query tiles of the entries with several tokens
(tensor-core prompt attention), the rows of those with one (split-KV decode attention) and the run of
rows of every entry (recurrent layers). For latent attention also the pages of the contexts whose keys
and values are expanded, and the rows that attend to the latents directly. Everything travels in one
pinned copy."""
from __future__ import annotations

from dataclasses import dataclass
from typing import List, Optional, Sequence

import torch

TILE_ROWS = 128


@dataclass
class Entry:
    """The next tokens of one sequence and the places among them whose logits are wanted."""
    seq_id: int
    tokens: Sequence[int]
    want: Sequence[int] = ()


def query_tiles(starts: Sequence[int], lens: Sequence[int], pos0: Sequence[int], slots: Sequence[int],
                tile_rows: int = TILE_ROWS) -> List[tuple]:
    """(first row, rows, position of the first row, table row) of every query tile of the entries with
    more than one token, the tiles that see most keys first."""
    tiles = []
    for start, n, pos, slot in zip(starts, lens, pos0, slots):
        if n < 2:
            continue
        for lo in range(0, n, tile_rows):
            tiles.append((start + lo, min(tile_rows, n - lo), pos + lo, slot))
    tiles.sort(key=lambda t: -(t[2] + t[1]))
    return tiles


def query_lanes(lens: Sequence[int], heads: int, sm_count: int = 148) -> int:
    """Query tiles of 128 rows a block of the prompt attention takes: 2 (two softmax warps per
    scheduler, shared key / value tiles) when blocks of 256 rows still fill the machine and few of
    their second tiles are empty, else 1. The result does not depend on it."""
    tiles = sum(-(-n // TILE_ROWS) for n in lens if n > 1)
    pairs = sum(-(-n // (2 * TILE_ROWS)) for n in lens if n > 1)
    return 2 if pairs * heads >= sm_count and tiles >= 1.5 * pairs else 1


class RaggedBatch:
    """``plan`` is host arithmetic; ``upload`` puts the arrays on the cache's device."""

    def __init__(self, entries: Sequence[Entry], pos0: Sequence[int], slots: Sequence[int], heads: int = 1,
                 absorb: Optional[int] = None, page: int = 16):
        """``absorb``: for latent attention, entries of up to this many tokens attend to the latents (their
        rows are listed one by one), the others to keys and values expanded for their whole context."""
        if not entries or any(len(e.tokens) < 1 for e in entries):
            raise ValueError("a batch needs at least one entry, and every entry at least one token")
        if len({e.seq_id for e in entries}) != len(entries):
            raise ValueError("a sequence appears twice in one batch")
        self.entries = list(entries)
        self.lens = [len(e.tokens) for e in entries]
        self.starts, n = [], 0
        for l in self.lens:
            self.starts.append(n)
            n += l
        self.num_tokens = n
        self.pos0, self.slots = list(pos0), list(slots)
        self.lanes = query_lanes(self.lens, heads)
        self.tiles_host = query_tiles(self.starts, self.lens, self.pos0, self.slots, TILE_ROWS * self.lanes)
        self.single_host = [s for s, l in zip(self.starts, self.lens) if l == 1]
        self.want_host = [s + w for s, e, l in zip(self.starts, self.entries, self.lens) for w in e.want]
        for e, l in zip(self.entries, self.lens):
            if any(not 0 <= w < l for w in e.want):
                raise ValueError("wanted place outside the entry's tokens")
        # longest context a single-token row sees (plans its KV splits)
        self.single_len = max([p + 1 for p, l in zip(self.pos0, self.lens) if l == 1], default=0)
        self.tokens: Optional[torch.Tensor] = None
        # latent attention: (table row, page) of every expanded page, tiles over them with the first
        # context row of their sequence, and the absorbed rows
        self.ctx_pages_host: List[tuple] = []
        self.latent_tiles_host: List[tuple] = []
        self.tile_ctx_host: List[int] = []
        self.absorbed_host: List[int] = []
        self.absorbed_len = 0
        if absorb is not None:
            wide = [i for i, l in enumerate(self.lens) if l > absorb]
            pick = lambda v: [v[i] for i in wide]                         # noqa: E731
            self.latent_lanes = query_lanes(pick(self.lens), heads)
            self.latent_tiles_host = query_tiles(pick(self.starts), pick(self.lens), pick(self.pos0), pick(self.slots),
                                                 TILE_ROWS * self.latent_lanes)
            first = {}
            for i in wide:
                first[self.slots[i]] = len(self.ctx_pages_host) * page
                self.ctx_pages_host += [(self.slots[i], p) for p in range(-(-(self.pos0[i] + self.lens[i]) // page))]
            self.tile_ctx_host = [first[t[3]] for t in self.latent_tiles_host]
            narrow = [i for i, l in enumerate(self.lens) if l <= absorb]
            self.absorbed_host = [self.starts[i] + j for i in narrow for j in range(self.lens[i])]
            self.absorbed_len = max([self.pos0[i] + self.lens[i] for i in narrow], default=0)

    @staticmethod
    def plan(entries: Sequence[Entry], cache, heads: int = 1, absorb: Optional[int] = None) -> "RaggedBatch":
        """Positions and table rows from the cache's current state; ``heads``: query heads of the
        model (of its narrowest layer), which with the lengths decides the tile height."""
        return RaggedBatch(entries, [cache.seq_len(e.seq_id) for e in entries],
                           [cache.slot_of[e.seq_id] for e in entries], heads, absorb, cache.block_size)

    def upload(self, device) -> "RaggedBatch":
        n, tiles = self.num_tokens, self.tiles_host
        runs = [x for s, l, slot, p in zip(self.starts, self.lens, self.slots, self.pos0) for x in (s, l, slot, p)]
        parts = [torch.tensor([x for t in tiles for x in t], dtype=torch.int32),     # 16-byte records first
                 torch.tensor(runs, dtype=torch.int32),
                 torch.tensor([x for t in self.latent_tiles_host for x in t], dtype=torch.int32),
                 torch.tensor([x for t in self.ctx_pages_host for x in t], dtype=torch.int32),   # 8-byte records
                 torch.tensor(self.tile_ctx_host, dtype=torch.int32),
                 torch.tensor(self.absorbed_host, dtype=torch.int32),
                 torch.cat([torch.as_tensor(e.tokens, dtype=torch.int32).reshape(-1) for e in self.entries]),
                 torch.cat([torch.arange(p, p + l, dtype=torch.int32) for p, l in zip(self.pos0, self.lens)]),
                 torch.repeat_interleave(torch.tensor(self.slots, dtype=torch.int32), torch.tensor(self.lens)),
                 torch.tensor(self.single_host, dtype=torch.int32),
                 torch.tensor(self.want_host, dtype=torch.int32)]
        flat = torch.cat(parts)
        device = torch.device(device)
        if device.type == "cuda":
            flat = flat.pin_memory().to(device, non_blocking=True)
        out, at = [], 0
        for p in parts:
            out.append(flat[at:at + p.numel()])
            at += p.numel()
        self.tiles = out[0].view(-1, 4) if tiles else None
        self.runs = out[1].view(-1, 4)            # (first row, rows, slot, position of the first row) per entry
        self.latent_tiles = out[2].view(-1, 4) if self.latent_tiles_host else None
        self.ctx_pages, self.tile_ctx = out[3].view(-1, 2), out[4]
        self.absorbed = out[5] if self.absorbed_host else None
        self.tokens, self.positions, self.token_seq = out[6], out[7], out[8]
        self.single = out[9] if self.single_host else None
        self.want = out[10]
        assert self.tokens.numel() == n
        return self
