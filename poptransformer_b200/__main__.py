"""Command line: greedy generation with any model of the registry.

    python -m poptransformer_b200 generate --model DIR --prompt 5,17,3 --prompt 9,4 --new 32

--model is a folder with config.json and weights; every --prompt (token ids) is one row of the batch.  Prints one JSON line per
row with its ids."""
import argparse
import json

import numpy as np


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m poptransformer_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="greedy generation from token ids")
    g.add_argument("--model", required=True, help="folder with config.json and weight files")
    g.add_argument("--prompt", action="append", required=True, help="token ids, comma separated; repeat for more rows")
    g.add_argument("--new", type=int, default=16, help="tokens to generate after the longest prompt")
    g.add_argument("--dtype", default=None, help="element type (default: the architecture's first)")
    g.add_argument("--eos", type=int, default=-1, help="end id: generation stops once every row has produced it")
    g.add_argument("--prefill", action="store_true", help="ingest the prompts in one pass where the decoder can")
    args = ap.parse_args(argv)
    from . import registry
    prompts = [[int(x) for x in p.split(",")] for p in args.prompt]
    max_len = max(map(len, prompts)) + args.new
    dec = registry.load_decoder(args.model, len(prompts), max_len, args.dtype, pad_id=-1, eos_id=args.eos, early_stop=args.eos >= 0)
    ids = np.full((len(prompts), max_len), -1, dtype=np.int32)
    for r, p in enumerate(prompts):
        ids[r, :len(p)] = p
    out = dec.run(ids, max_loop=max_len - 1, prefill=args.prefill and hasattr(dec, "prefill"))["Loop:0"]
    for row in out:
        print(json.dumps({"ids": [int(t) for t in row if t >= 0]}))


if __name__ == "__main__":
    main()
