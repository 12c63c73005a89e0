"""Replay a recorded schedule of token portions through a model and write the logits it asks for.

    bin/trace_run --model DIR --dtype bfloat16 --out OUT --max-tokens 4096 < steps.jsonl

One JSON object per line on standard input is one engine step (``engine.session.Session.feed``):

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

``entries`` name each request's next tokens and the places among them whose logits are wanted, ``end`` the requests that are
finished after the step. A step that wants something writes ``OUT/<step>.f32`` (little-endian fp32 ``[wanted, vocab]``, in the
order of the entries). ``done <step>`` is printed after every step. ``--dtype float32`` runs models that have a true fp32 path.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
from typing import List, Optional

SLOTS = 64


def main(argv: Optional[List[str]] = None) -> int:
    ap = argparse.ArgumentParser(description="Feed recorded steps to a model and write the logits they ask for")
    ap.add_argument("--model", required=True, help="directory with config.json and safetensors weights")
    ap.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    ap.add_argument("--out", required=True, help="directory for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=4096, help="most tokens all live requests hold at any time")
    args = ap.parse_args(argv)

    import numpy as np
    import torch

    from ..models.registry import load_model
    from ..ops import kernels as K
    from .generation import PAGE, Generator, page_elems
    from .session import Session

    torch.cuda.set_device(0)
    dev = torch.device("cuda:0")
    dtype = getattr(torch, args.dtype)
    seq = -(-max(args.max_tokens, PAGE) // PAGE) * PAGE
    model = load_model(args.model, dev, dtype=dtype, max_pos=seq)
    # every live request wastes less than one page, plus the scratch page
    pages = seq // PAGE + SLOTS + 1
    gen = Generator(model, max_slots=SLOTS, max_seq_len=seq, kv_budget_bytes=pages * page_elems(model.cfg.kv_geometry()) * dtype.itemsize,
                    use_graphs=False)
    session = Session(gen)
    os.makedirs(args.out, exist_ok=True)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(e["id"], e["tokens"], e.get("want", [])) for e in step["entries"]]
        got = [t for t in session.feed(entries) if t is not None]
        if got:
            logits = torch.cat([t.float() for t in got]).cpu().numpy().astype("<f4", copy=False)
            path = os.path.join(args.out, f"{step['step']}.f32")
            np.ascontiguousarray(logits).tofile(path)
        for rid in step.get("end", []):
            session.end(rid)
        K.check_status()
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
