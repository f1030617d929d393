"""Generation from the command line, for every architecture in the registry.

    python -m async_grpo_nccl_b200.generate --model DIR|preset --prompt-ids 5,17,3 --max-new-tokens 32
    python -m async_grpo_nccl_b200.generate --model DIR --prompts prompts.jsonl --n 4 --temperature 0.8 --logprobs

Prompts are token ids (``--prompt-ids``, repeatable, or JSONL rows with ``input_token_ids``) or, when the model directory
holds a tokenizer, text (``--prompt``, or rows with ``input``). All prompts go to the engine at once; each finished sample
is one JSON line on standard output.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import Any, List, Optional, Sequence


def read_prompts(args: argparse.Namespace, tokenizer: Any) -> List[List[int]]:
    def encode(text: str) -> List[int]:
        if tokenizer is None:
            raise SystemExit("text prompts need a tokenizer in the model directory; pass token ids instead")
        return list(tokenizer.encode(text, add_special_tokens=False))

    out = [[int(t) for t in p.split(",")] for p in args.prompt_ids] + [encode(p) for p in args.prompt]
    if args.prompts:
        with open(args.prompts, "r", encoding="utf-8") as f:
            for line in f:
                if line.strip():
                    row = json.loads(line)
                    out.append([int(t) for t in row["input_token_ids"]] if "input_token_ids" in row else encode(row["input"]))
    return out


def main(argv: Optional[Sequence[str]] = None) -> int:
    ap = argparse.ArgumentParser(prog="async_grpo_nccl_b200.generate")
    ap.add_argument("--model", required=True, help="model directory (config.json + safetensors) or preset name (random weights)")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--prompt-ids", action="append", default=[], help="comma-separated token ids (repeatable)")
    ap.add_argument("--prompt", action="append", default=[], help="text (repeatable)")
    ap.add_argument("--prompts", default=None, help="JSONL file, one prompt per row")
    ap.add_argument("--n", type=int, default=1, help="samples per prompt")
    ap.add_argument("--max-new-tokens", type=int, default=64)
    ap.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--ignore-eos", action="store_true")
    ap.add_argument("--logprobs", action="store_true", help="also print the log-probability of every sampled token")
    ap.add_argument("--max-seqs", type=int, default=256)
    ap.add_argument("--max-model-len", type=int, default=None)
    ap.add_argument("--max-prefill-tokens", type=int, default=16384)
    ap.add_argument("--kv-gb", type=float, default=None, help="memory for the KV cache (default: 60 %% of what is free)")
    ap.add_argument("--cuda-graphs", action="store_true", help="capture the decode step")
    args = ap.parse_args(argv)
    from .serving import load_engine

    tokenizer = None
    if os.path.isdir(args.model) and any(f.startswith("tokenizer") for f in os.listdir(args.model)):
        from transformers import AutoTokenizer

        tokenizer = AutoTokenizer.from_pretrained(args.model)
    prompts = read_prompts(args, tokenizer)
    if not prompts:
        ap.error("no prompts")
    max_len = args.max_model_len or max(len(p) for p in prompts) + args.max_new_tokens + 1
    eng = load_engine(args.model, args.dtype, seed=args.seed, max_model_len=max_len, max_seqs=max(args.max_seqs, args.n),
                      max_prefill_tokens=args.max_prefill_tokens, use_cuda_graph=args.cuda_graphs,
                      kv_memory_bytes=int(args.kv_gb * 2 ** 30) if args.kv_gb else None)
    if args.logprobs:
        eng.enable_logprobs()
    for i, p in enumerate(prompts):
        eng.add_request(i, p, n=args.n, max_new_tokens=args.max_new_tokens, temperature=args.temperature, seed=args.seed + i,
                        ignore_eos=args.ignore_eos)
    done = eng.run_until_done()
    eng.check_status()
    for f in sorted(done, key=lambda f: (f.request_id, f.child)):
        row = {"prompt": f.request_id, "sample": f.child, "finish_reason": f.finish_reason, "output_token_ids": [int(t) for t in f.output_ids]}
        if tokenizer is not None:
            row["text"] = tokenizer.decode(row["output_token_ids"])
        if args.logprobs:
            row["logprobs"] = [float(x) for x in f.output_logprobs]
        print(json.dumps(row), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
