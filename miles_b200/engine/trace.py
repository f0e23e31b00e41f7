"""Replay a trace of given token ids through the engine, step by step, and write the logits asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N

Standard input has one JSON object per line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

Each entry's tokens continue that request from the cache and state earlier steps left; all entries of a step are one batch
(`Engine.feed`).  Logits at the wanted places go to OUT/<step>.f32 (little-endian float32, [wanted, vocab]); a line
`done <step>` follows every step.  Requests in `end` give back their blocks and state slot.  Nothing is sampled.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

SLOTS = 4          # requests that may be live at once


def main(argv=None) -> int:
    p = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    p.add_argument("--model", required=True, help="folder with config.json and safetensors weights")
    p.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    p.add_argument("--out", required=True)
    p.add_argument("--max-tokens", type=int, required=True, help="tokens the live requests hold at most, each rounded up to the page size")
    p.add_argument("--block-size", type=int, default=64, help="tokens per cache page")
    a = p.parse_args(argv)

    import torch

    from ..ops import build

    if not torch.cuda.is_available():
        print("trace replay runs the CUDA kernels: no CUDA device found", file=sys.stderr)
        return 2
    from ..models.config import get_config

    cfg = get_config(a.model)
    build.build_serve(build.serve_kind(cfg))
    from .engine import Engine

    # a true 32-bit run: no TF32 in the dense projections
    torch.backends.cuda.matmul.allow_tf32 = False
    torch.cuda.set_device(0)
    engine = Engine(cfg, device="cuda:0", dtype=getattr(torch, a.dtype), num_blocks=max(1, -(-a.max_tokens // a.block_size)), block_size=a.block_size,
                    max_running_requests=SLOTS, max_context_len=max(a.max_tokens, a.block_size), prefix_cache=False)
    engine.update_weights_from_disk(a.model)
    replay(engine, sys.stdin, a.out)
    return 0


def replay(engine, lines, out_dir: str, answer=lambda s: print(s, flush=True)):
    live: dict = {}
    os.makedirs(out_dir, exist_ok=True)
    for line in lines:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in live:
                live[e["id"]] = engine.open_request(str(e["id"]))
            entries.append((live[e["id"]], list(e["tokens"]), list(e["want"])))
        if entries:
            logits = engine.feed(entries)
            if logits.shape[0]:
                path = os.path.join(out_dir, f"{step['step']}.f32")
                with open(path + ".part", "wb") as f:
                    f.write(logits.cpu().numpy().astype("<f4").tobytes())
                os.replace(path + ".part", path)
        for rid in step.get("end", []):
            live.pop(rid)
            engine.close_request(str(rid))
        answer(f"done {step['step']}")


if __name__ == "__main__":
    sys.exit(main())
