"""Cached decode of models with a layer list of their own (``models/ragged_model.py``): one row per sequence, one CUDA
graph per step. Up to ``MATVEC_ROWS`` rows a family's mat-vec form runs (``_matvec_layers``) where its layers fit it
(``_fits``); larger batches, head sizes outside the fused attention kernel and 32-bit models run the layers of the
ragged batch with every row a sequence of its own, captured the same way."""
from __future__ import annotations

from typing import Optional

import torch

from .. import _lib
from ..ops import parallel_block as P
from ..ops import post_norm as N
from .decode_engine import DecodeEngineBase
from .ragged_model import Buffers, RaggedModel, StepContext

# Above this many rows the GEMM form of the step runs.
MATVEC_ROWS = 3


class LayeredDecode(DecodeEngineBase):
    def __init__(self, model: RaggedModel, cache, max_batch: int = 1, use_graph: bool = True, pdl: bool = True,
                 greedy: bool = True, matvec_rows: int = MATVEC_ROWS):
        super().__init__(model, cache, max_batch, use_graph, pdl, greedy)
        self.bufs = Buffers(max_batch, model.device)
        self.matvec_rows = matvec_rows
        self.max_len = cache.max_blocks_per_seq * cache.block_size
        self._planned = set()
        self.ticket = torch.zeros(1, dtype=torch.int32, device=model.device)
        self.fused = model.dtype == torch.bfloat16 and P.gemv_max_rows(model.width_p) > 0 and \
            N.max_rows(model.width_p) > 0 and all(self._fits(lw) for lw in model.w.layers)

    def _fits(self, lw) -> bool:
        """Whether the layer has a mat-vec form: staged rows fit shared memory, head sizes the attention kernel."""
        return False

    def _matvec_layers(self, c: StepContext) -> None:
        """The whole step in mat-vec form, from the embedding to the logits."""
        raise NotImplementedError

    def capture(self, nb: Optional[int] = None):
        """Buffers and scratch of a bucket come with its first run: one plain run first, so that the recorded
        step allocates nothing (which the native graph store asks for)."""
        nb = self.bucket() if nb is None else nb
        if nb not in self._planned:
            self._planned.add(nb)
            restore = self._snapshot()
            self._run_step(nb)
            restore()
        return super().capture(nb)

    def _context(self, nb: int) -> StepContext:
        return StepContext(nb, self.bufs, self.cache, self.block_table[:nb], self.positions[:nb], None,
                           None if self.state_slots is None else self.state_slots[:nb], None, None, self.max_len, self.pdl)

    def _run_step(self, nb: Optional[int] = None) -> None:
        m = self.model
        nb = self.B if nb is None else nb
        n0 = _lib.launch_count()
        c = self._context(nb)
        if self.fused and nb <= self.matvec_rows:
            self._matvec_layers(c)
        else:
            acts = m.start(self.tokens[:nb], self.bufs)
            for li in range(len(m.w.layers)):
                m.layer(li, acts, c)
            m.logits(acts[0], acts[1], out=self.logits[:nb], pdl=self.pdl)
        self._finish_step(pdl=self.pdl and m.dtype == torch.bfloat16, n0=n0, nb=nb)
