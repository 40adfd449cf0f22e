"""Generates token ids from a prompt of token ids.

    python -m onellm_b200.generate --model DIR --prompt 5,17,3 [--prompt ...] --new 16 [--top-k K] [--temperature T]
                                   [--dtype bfloat16|float32] [--max-seq-len S] [--weights PREFIX]

DIR is a model folder: config.json + model.safetensors (the design is named in config.json), or the config.ini of a
converted LLaMA checkpoint, whose weight files --weights names by their prefix (default DIR/).  Several prompts, of any
lengths, are decoded as one batch; one line of ids is printed per prompt.
"""
from __future__ import annotations

import argparse
import os
import sys


def open_any(folder, weights=None, dtype="bfloat16", max_batch=1, max_seq_len=0):
    """The engine for a model folder of either kind."""
    import onellm_b200 as ob
    ini = os.path.join(folder, "config.ini")
    if not os.path.exists(os.path.join(folder, "config.json")) and os.path.exists(ini):
        m = ob.Llama.from_ini(ini, max_batch, max_seq_len)
        m.load_weights(weights or os.path.join(folder, ""))
        return m
    return ob.open_model(folder, ob.F32 if dtype == "float32" else ob.BF16, max_batch, max_seq_len)


def generate(model, prompts, n_new):
    """n_new ids behind every prompt (a list of id lists), int32 [len(prompts), n_new]."""
    import numpy as np
    out = np.zeros((len(prompts), n_new), np.int32)
    if n_new == 0:
        return out
    out[:, 0] = model.prefill_ragged(prompts)
    ids = np.zeros(len(prompts), np.int32)
    for t in range(1, n_new):
        model.decode_step(out_ids=ids)
        out[:, t] = ids
    return out


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m onellm_b200.generate")
    ap.add_argument("--model", required=True)
    ap.add_argument("--weights", help="prefix of a converted LLaMA checkpoint's weight files")
    ap.add_argument("--prompt", action="append", required=True, help="token ids with commas between them")
    ap.add_argument("--new", type=int, default=16)
    ap.add_argument("--top-k", type=int, default=1)
    ap.add_argument("--temperature", type=float, default=1.0)
    ap.add_argument("--dtype", choices=["bfloat16", "float32"], default="bfloat16")
    ap.add_argument("--max-seq-len", type=int, default=0)
    args = ap.parse_args(argv)
    prompts = [[int(x) for x in p.split(",")] for p in args.prompt]
    m = open_any(args.model, args.weights, args.dtype, len(prompts), args.max_seq_len)
    m.set_sampling(args.top_k, args.temperature)
    for row in generate(m, prompts, args.new):
        print(",".join(str(int(i)) for i in row))
    m.close()
    return 0


if __name__ == "__main__":
    sys.exit(main())
