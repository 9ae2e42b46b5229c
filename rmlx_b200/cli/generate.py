"""``rmlx_b200 generate``: run prompts of token ids through the serving engine (continuous batching,
paged cache, the family's kernels) and print the generated ids, one JSON object.

    python -m rmlx_b200.cli generate --model DIR --prompt 1,2,3 --prompt 7,8 --steps 16
        [--dtype bfloat16|float32] [--temperature 0.8 --top-k 40 --top-p 0.95 --seed 1] [--eos ID]"""
from __future__ import annotations

import argparse
import json
from typing import Optional, Sequence


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="rmlx_b200 generate")
    ap.add_argument("--model", required=True, help="checkpoint folder (config.json, safetensors)")
    ap.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; may be repeated")
    ap.add_argument("--steps", type=int, default=16, help="tokens to generate per prompt")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--device", default=None, help="default: cuda if there is one")
    ap.add_argument("--temperature", type=float, default=0.0, help="0: greedy")
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--repetition-penalty", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=None)
    ap.add_argument("--eos", type=int, default=-1, help="stop token")
    ap.add_argument("--chunk", type=int, default=512, help="prompt tokens per step")
    ap.add_argument("--max-batch", type=int, default=8, help="sequences decoded together")
    a = ap.parse_args(argv)
    prompts = [[int(t) for t in p.split(",")] for p in a.prompt]

    import torch
    from ..config import SamplerConfig, SchedulerConfig
    from ..kv.paged import PAGE
    from ..models.registry import from_pretrained
    from ..serve.engine import ServingEngine
    device = a.device or ("cuda" if torch.cuda.is_available() else "cpu")
    model = from_pretrained(a.model, device, getattr(torch, a.dtype))
    blocks = 2 + sum((len(p) + a.steps) // PAGE + 1 for p in prompts)
    engine = ServingEngine(model, blocks,
                           SchedulerConfig(max_batch_size=min(a.max_batch, len(prompts)), max_prefill_chunk=a.chunk,
                                           eos_token_id=a.eos),
                           SamplerConfig(a.temperature, a.top_k, a.top_p, a.repetition_penalty, a.seed))
    ids = [engine.submit(p, a.steps) for p in prompts]
    out = engine.run_until_done()
    print(json.dumps({"tokens": [out[i] for i in ids]}))
    return 0
