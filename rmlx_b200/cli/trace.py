"""``rmlx_b200 trace-run`` (also ``bin/trace_run``): replay given token ids through a model, step by
step, and write logits. It samples nothing; it drives the serving engine's own step
(``ServingEngine.run_entries``), cache and kernels.

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries``: for each request its next tokens and the places among them whose logits are wanted;
``end``: the requests whose pages and slot are given back after the step. A step with wanted logits
writes ``<out>/<step>.f32`` (little-endian fp32, [wanted, vocab], in the order of the entries and of
``want``); after every step ``done <step>`` is printed."""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional, Sequence

SLOTS = 4            # requests that may be live at any time
DTYPES = ("bfloat16", "float32")


class TraceReplay:
    """Requests by name on top of a serving engine."""

    def __init__(self, engine):
        self.engine = engine
        self.seq_of: Dict[str, int] = {}

    def step(self, entries: Sequence[dict], end: Sequence[str] = ()):
        """Runs one step; returns the wanted logits on the host (None when nothing is wanted)."""
        from ..models.ragged import Entry
        batch = []
        for e in entries:
            if e["id"] not in self.seq_of:
                self.seq_of[e["id"]] = self.engine.open_sequence()
            batch.append(Entry(self.seq_of[e["id"]], e["tokens"], e.get("want", ())))
        logits = None
        if batch:
            out = self.engine.run_entries(batch)
            if any(len(e.want) for e in batch):
                logits = out.float().cpu()
        for name in end:
            self.engine.close_sequence(self.seq_of.pop(name))
        return logits


def make_engine(model_dir: str, dtype: str, max_tokens: int, device="cuda"):
    """Serving engine whose page pool holds ``max_tokens`` tokens (page 0 is reserved) and that has
    ``SLOTS`` sequence slots."""
    import torch
    from ..config import SchedulerConfig
    from ..kv.paged import PAGE
    from ..models.registry import from_pretrained
    from ..ops.gemm import GemmStatus
    from ..serve.engine import ServingEngine
    if dtype == "float32":          # library products of the models that use them stay in 32-bit, too
        torch.backends.cuda.matmul.allow_tf32 = False
        torch.backends.cudnn.allow_tf32 = False
    model = from_pretrained(model_dir, device, getattr(torch, dtype))
    blocks = (max_tokens + PAGE - 1) // PAGE + 1
    engine = ServingEngine(model, blocks, SchedulerConfig(max_batch_size=SLOTS))
    return engine, lambda: GemmStatus.check(model.device)


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="replay token ids through a model and write logits")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=DTYPES)
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="tokens that live requests hold at most")
    a = ap.parse_args(argv)
    engine, check = make_engine(a.model, a.dtype, a.max_tokens)
    replay = TraceReplay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        logits = replay.step(step.get("entries", ()), step.get("end", ()))
        if logits is not None:
            check()
            path = os.path.join(a.out, f"{step['step']}.f32")
            with open(path, "wb") as f:
                f.write(logits.numpy().astype("<f4").tobytes())
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
