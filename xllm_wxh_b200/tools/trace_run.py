"""Replay recorded token streams through the engine (`bin/trace_run`).

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps.jsonl

Every input line is one engine step:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Its entries run as one batch: the next tokens of each named request, behind what earlier steps left in the cache.  `want`
lists places among those tokens; their logits go to <out>/<step>.f32 as little-endian fp32 [wanted, vocab], entry by entry.
Requests under `end` are over after the step and give their blocks and state slots back.  `done <step>` is printed when a step is complete.
Nothing is sampled; batches, blocks, kernels and CUDA graphs are those of generation (`LLMEngine.step_portions`).
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, List, Optional

BLOCK = 64          # tokens per KV block
LIVE = 4            # requests that may hold recurrent state at a time, in models that keep any


def main(argv: Optional[List[str]] = None) -> int:
    p = argparse.ArgumentParser(prog="trace_run", description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    p.add_argument("--model", required=True, help="model directory (config.json, *.safetensors)")
    p.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16",
                   help="bfloat16: as the model is served; float32: everything in true 32-bit")
    p.add_argument("--out", required=True, help="directory of the logit files")
    p.add_argument("--max-tokens", type=int, required=True,
                   help=f"most tokens that live requests hold at any time (each rounded up to {BLOCK}): size of the KV cache")
    p.add_argument("--device", default="cuda:0")
    a = p.parse_args(argv)

    import numpy as np
    from ..config import Options
    from ..runtime.engine import LLMEngine
    blocks = (a.max_tokens + BLOCK - 1) // BLOCK
    engine = LLMEngine(Options(model=a.model, devices=a.device, dtype=a.dtype, block_size=BLOCK, num_kv_blocks=blocks + 1, num_state_slots=LIVE,
                               max_tokens_per_batch=max(64, a.max_tokens), max_seqs_per_batch=64, enable_prefix_cache=False,
                               max_model_len=max(64, blocks * BLOCK), enable_numa_binding=False))
    os.makedirs(a.out, exist_ok=True)
    live: Dict[str, int] = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        portions = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.add_request([])
            portions.append((live[e["id"]], e["tokens"], e.get("want", [])))
        rows = [r for r in engine.step_portions(portions) if len(r)]
        if rows:
            path = os.path.join(a.out, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(np.ascontiguousarray(np.concatenate(rows), dtype="<f4").tobytes())
            os.replace(path + ".part", path)
        for i in step.get("end", []):
            engine.cancel(live.pop(i))
        print(f"done {step['step']}", flush=True)
    if engine.device.type == "cuda":
        from ..ops import cuda_ops
        status = cuda_ops.read_status()
        if status:
            print(f"a kernel reported status {status}", file=sys.stderr)
            return 1
    engine.shutdown()
    return 0
