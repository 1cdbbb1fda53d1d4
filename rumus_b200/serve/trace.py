"""Trace runner: pushes given token ids through a model step by step and writes logits.

    python -m rumus_b200.serve.trace --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

``DIR`` holds ``config.json`` and ``model.safetensors``.  Steps come on standard input, one JSON object a line:

    {"step": 7, "entries": [{"id": "x", "tokens": [11, 4], "want": [1]}, {"id": "y", "tokens": [9], "want": [0]}], "end": ["y"]}

All entries of a step are one batch.  The logits at the wanted places go to ``OUT/<step>.f32`` (little-endian,
``[wanted, vocab]``, in the order of the entries), and ``done <step>`` is printed after every step.  The cache
pool holds ``--max-tokens`` tokens of live sequences; ``end`` names the sequences that give theirs back.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__.splitlines()[0])
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens live sequences hold at any time")
    ap.add_argument("--max-live", type=int, default=4, help="most sequences alive at any time")
    a = ap.parse_args(argv)

    from ..models.registry import architecture, read_config_json
    from .. import build
    from ..ops import _lib
    _lib.use_part(build.ensure(architecture(read_config_json(a.model)["architecture"]).parts))

    import torch
    from .loading import load_engine
    bs = 64
    engine = load_engine(a.model, torch.device("cuda", 0), getattr(torch, a.dtype), block_size=bs,
                         num_blocks=(a.max_tokens + bs - 1) // bs, max_batch=a.max_live, max_seq_len=a.max_tokens)
    rids, next_rid = {}, 0
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        portions = []
        for e in step["entries"]:
            if e["id"] not in rids:
                next_rid += 1
                rids[e["id"]] = next_rid
            portions.append((rids[e["id"]], e["tokens"], e.get("want", [])))
        logits = engine.feed(portions) if portions else None
        if logits is not None:
            with open(os.path.join(a.out, f"{step['step']}.f32"), "wb") as f:
                f.write(logits.float().cpu().numpy().astype("<f4").tobytes())
        for i in step.get("end", []):
            engine.release(rids.pop(i))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
