"""Greedy generation from a model folder, token ids in and out.

    python -m vesper_b200.generate --model DIR --prompt "5 17 3" [--prompt ...] [--new N] [--dtype bfloat16|float32] [--stop ID ...]

The folder holds config.json and model.safetensors; the model class comes from the configuration's "architecture".
Prompts of one call have one length and run as a batch; one line of ids per prompt is printed.
"""
import argparse

import numpy as np


def main():
    ap = argparse.ArgumentParser(description=__doc__, formatter_class=argparse.RawDescriptionHelpFormatter)
    ap.add_argument("--model", required=True)
    ap.add_argument("--prompt", action="append", required=True, help="token ids, separated by blanks")
    ap.add_argument("--new", type=int, default=32, help="tokens to generate")
    ap.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    ap.add_argument("--stop", type=int, nargs="*", default=[], help="ids that end a sequence")
    a = ap.parse_args()
    prompts = [[int(t) for t in p.split()] for p in a.prompt]
    if len({len(p) for p in prompts}) != 1 or not prompts[0]:
        ap.error("the prompts of a call must have one length")
    from .build import build_host
    build_host()
    from .model import load_model
    m = load_model(a.model, a.dtype, max_seq_len=len(prompts[0]) + a.new)
    toks, _ = m.generate_greedy(np.array(prompts, np.int32), a.new, stop_ids=a.stop)
    for row in toks:
        print(" ".join(str(t) for t in row))
    m.close()


if __name__ == "__main__":
    main()
