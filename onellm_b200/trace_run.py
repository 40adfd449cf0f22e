"""Replays given token ids through a model, step by step, and writes the logits that are asked for.

    bin/trace_run --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N  < steps

Steps come as JSON objects, one a line, on standard input:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

A step feeds the next tokens of one request and names the places among them whose logits are wanted; `end` lists the
requests that are over.  The logits of a step go to OUT/<step>.f32 as little-endian float32 [wanted, vocab]; `done
<step>` is printed after every step.  The engine is the one that generates: a request's first tokens are a prefill,
several further tokens an extension behind the cached positions, a single further token a decode step, and nothing is
sampled.  Requests run one after the other on one sequence of the engine, which is cleared for each.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


class TraceRunner:
    def __init__(self, model):
        self.model = model
        model.set_sampling(top_k=0)
        self.current = None  # the request that holds the sequence
        self.cached = 0
        self.over = set()

    def feed(self, request, tokens, want):
        """The next tokens of a request; float32 [len(want), vocab]."""
        import numpy as np
        if request != self.current:
            if request in self.over:
                raise ValueError(f"request {request!r} is over")
            if self.current is not None:
                self.end(self.current)
            self.current, self.cached = request, 0
        ids = np.asarray(tokens, np.int32)
        if self.cached and len(ids) == 1:
            self.model.decode_step(in_ids=ids)
            self.cached += 1
            if not want:
                self.model.sync()
                return None
            row = self.model.logits(1)
            return row[[0] * len(want)]
        if want:
            self.model.want_logits(want)
        if self.cached:
            self.model.extend(ids[None, :])
        else:
            self.model.prefill(ids[None, :])
        self.cached += len(ids)
        return self.model.row_logits(len(want)) if want else None

    def end(self, request):
        self.over.add(request)
        if request == self.current:
            self.current, self.cached = None, 0


def main(argv=None):
    ap = argparse.ArgumentParser(prog="trace_run", description="Replays token ids through a model and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--out", required=True, help="folder for <step>.f32")
    ap.add_argument("--max-tokens", type=int, default=0, help="most tokens a request holds (0: what the model allows)")
    args = ap.parse_args(argv)

    from onellm_b200 import build
    import onellm_b200 as ob
    ob.LIB_PATH = build.library_for(args.model)
    model = ob.open_model(args.model, ob.BF16 if args.dtype == "bfloat16" else ob.F32, max_batch=1, max_seq_len=args.max_tokens)
    run = TraceRunner(model)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        parts = []
        for e in step["entries"]:
            rows = run.feed(e["id"], e["tokens"], e["want"]) if e["tokens"] else None
            if rows is not None:
                parts.append(rows.astype("<f4").tobytes())
        if parts:
            with open(os.path.join(args.out, f"{step['step']}.f32"), "wb") as f:
                f.write(b"".join(parts))
        for r in step.get("end", []):
            run.end(r)
        print(f"done {step['step']}", flush=True)
    model.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
