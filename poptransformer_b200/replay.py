"""Replays a trace of batches through a model, step by step, and writes logits (no sampling).

Steps come on standard input, one JSON object a line:

    {"step": 0, "entries": [{"id": "a", "tokens": [5, 17, 3], "want": [0, 2]}], "end": []}

An entry brings the next tokens of a request (its first ones open it); `want` are the places among them whose logits are written
to OUT/<step>.f32 as little-endian float32 [places in order of the entries, vocab]; the requests in `end` are closed after the
step.  After every step the line `done <step>` is printed."""
import argparse
import json
import os
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(description="Replays a trace of batches and writes logits.")
    ap.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for the logits")
    ap.add_argument("--max-tokens", type=int, required=True, help="most tokens that open requests hold at any time")
    args = ap.parse_args(argv)

    from . import _lib, build, checkpoint, registry
    config, sd = checkpoint.load_model_dir(args.model)
    if args.dtype not in registry.dtypes(config):
        sys.stderr.write(f"{registry.architecture(config)} does not run in {args.dtype}\n")
        return 3
    _lib.use_library(build.build_for(registry.architecture(config)))
    page = 64
    dec, seqs = None, {}
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        fresh = [e["id"] for e in step["entries"] if e["id"] not in seqs]
        if dec is None:
            batch = len(fresh)
            dec = registry.build_decoder(config, sd, batch, args.max_tokens, args.dtype, page_size=page, n_pages=args.max_tokens // page + batch)
        elif not seqs and len(fresh) > dec.batch:
            dec.resize(len(fresh), n_pages=args.max_tokens // page + len(fresh))
        for i in fresh:
            seqs[i] = dec.open()
        logits = dec.extend([(seqs[e["id"]], e["tokens"], e["want"]) for e in step["entries"]])
        if logits.shape[0]:
            logits.cpu().numpy().astype("<f4").tofile(os.path.join(args.out, f"{step['step']}.f32"))
        for i in step["end"]:
            dec.close(seqs.pop(i))
        print(f"done {step['step']}", flush=True)
    return 0


if __name__ == "__main__":
    sys.exit(main())
