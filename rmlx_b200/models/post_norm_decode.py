"""Cached decode of post-norm decoders (``models/rodapel.py``): one row per sequence, one CUDA graph per
step. The layers are those of the ragged batch with every row a sequence of its own."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from .decode_engine import DecodeEngineBase
from .rodapel import Buffers, RodapelModel, StepContext


class PostNormDecode(DecodeEngineBase):
    def __init__(self, model: RodapelModel, cache, max_batch: int = 1, use_graph: bool = True, pdl: bool = True,
                 greedy: bool = True):
        super().__init__(model, cache, max_batch, use_graph, pdl, greedy)
        self.bufs = Buffers(max_batch, model.device)
        self.max_len = cache.max_blocks_per_seq * cache.block_size

    def _context(self, nb: int) -> StepContext:
        return StepContext(nb, self.bufs, self.cache, self.block_table[:nb], self.positions[:nb], None,
                           None if self.state_slots is None else self.state_slots[:nb], None, None, self.max_len, self.pdl)

    def _run_step(self, nb: Optional[int] = None) -> None:
        m = self.model
        nb = self.B if nb is None else nb
        n0 = _lib.launch_count()
        x, h = m.embed(self.tokens[:nb], self.bufs)
        c = self._context(nb)
        for li in range(len(m.w.layers)):
            m.layer(li, x, h, c)
        m.logits(x, h, out=self.logits[:nb], pdl=self.pdl)
        self._finish_step(pdl=self.pdl and m.dtype == torch.bfloat16, n0=n0, nb=nb)
