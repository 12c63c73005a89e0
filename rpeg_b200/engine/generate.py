"""Generate from a model directory of any supported family.

    python -m rpeg_b200.engine.generate --model DIR --prompt 5,17,3 --prompt 8,1 --max-new 32 --greedy
    python -m rpeg_b200.engine.generate --model DIR --prompts rows.jsonl --temperature 0.8 --top-p 0.9 --seed 7

Prompts are token ids: ``--prompt`` (comma separated, repeatable) or a JSONL file whose lines are lists of ids (or objects
with ``input_ids``). Prints one JSON object per prompt: its generated tokens and their log-probs.
"""
from __future__ import annotations

import argparse
import json
import sys
from typing import List, Optional


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(description="Generate token ids from a model directory")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors weights")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16", help="float32: families with a true fp32 path")
    ap.add_argument("--prompt", action="append", default=[], help="comma-separated token ids")
    ap.add_argument("--prompts", default=None, help="JSONL file of token id lists")
    ap.add_argument("--max-new", type=int, default=32)
    ap.add_argument("--greedy", action="store_true")
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--top-k", type=int, default=0)
    ap.add_argument("--top-p", type=float, default=1.0)
    ap.add_argument("--seed", type=int, default=0)
    ap.add_argument("--eos", type=int, default=-1, help="token id that ends a row (-1: none)")
    ap.add_argument("--slots", type=int, default=64, help="rows decoded together")
    ap.add_argument("--prefill-portion", type=int, default=0, help="most prompt tokens of a row per forward (0: whole prompts)")
    ap.add_argument("--kv-bytes", type=float, default=8e9)
    args = ap.parse_args(argv)

    prompts = [[int(t) for t in p.split(",")] for p in args.prompt]
    if args.prompts:
        with open(args.prompts) as f:
            rows = [json.loads(line) for line in f if line.strip()]
        prompts += [list(r["input_ids"] if isinstance(r, dict) else r) for r in rows]
    if not prompts or not all(prompts):
        ap.error("give at least one prompt, none of them empty")

    import torch

    from ..models.registry import load_model
    from ..ops import kernels as K
    from .generation import Generator

    dev = torch.device("cuda:0")
    torch.cuda.set_device(0)
    longest = max(len(p) for p in prompts) + args.max_new
    model = load_model(args.model, dev, dtype=getattr(torch, args.dtype), max_pos=longest)
    if max(max(p) for p in prompts) >= model.cfg.vocab or min(min(p) for p in prompts) < 0:
        ap.error(f"prompt tokens must lie in [0, {model.cfg.vocab})")
    gen = Generator(model, max_slots=min(args.slots, max(1, len(prompts))), max_seq_len=longest, kv_budget_bytes=args.kv_bytes, eos_id=args.eos,
                    prefill_portion=args.prefill_portion)
    res = gen.generate([torch.tensor(p, dtype=torch.int32) for p in prompts], args.max_new, temperature=args.temperature, greedy=args.greedy,
                       seed=args.seed, top_k=args.top_k, top_p=args.top_p)
    K.check_status()
    toks, lps, lens = res.tokens.tolist(), res.logprobs.tolist(), res.lengths.tolist()
    for i, n in enumerate(lens):
        print(json.dumps({"row": i, "tokens": toks[i][:n], "logprobs": [round(v, 5) for v in lps[i][:n]]}), flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
