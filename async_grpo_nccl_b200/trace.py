"""Trace replay: feeds given tokens through an engine's step-wise interface and writes the logits that are asked for.

It samples nothing. Model class, weights, cache, scheduler and kernels are the ones that generation uses: a step whose entry
has one token of a sequence that has begun is a decode step, anything else a (portion of a) prompt.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Dict, Optional, Sequence


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description=__doc__)
    ap.add_argument("--model", required=True, help="directory with config.json and model.safetensors")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that live requests hold at any time")
    ap.add_argument("--max-seqs", type=int, default=32, help="most requests alive at any time")
    args = ap.parse_args(argv)
    from .serving import UnsupportedDtype, load_engine

    max_len = args.max_tokens + 16
    try:
        eng = load_engine(args.model, args.dtype, max_seqs=args.max_seqs, max_model_len=max_len,
                          num_blocks=(args.max_tokens + 15) // 16 + args.max_seqs + 8)
    except UnsupportedDtype as e:
        print(e, file=sys.stderr)
        return 3
    ids: Dict[str, int] = {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = []
        for e in step["entries"]:
            if e["id"] not in ids:
                ids[e["id"]] = eng.open_sequence()
            if e["tokens"]:
                entries.append((ids[e["id"]], e["tokens"], e.get("want", [])))
        logits = eng.extend(entries) if entries else None
        if logits is not None and logits.shape[0]:
            data = logits.float().cpu().contiguous().numpy().astype("<f4")
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(data.tobytes())
        eng.check_status()
        for rid in step.get("end", []):
            if rid in ids:
                eng.close_sequence(ids.pop(rid))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
