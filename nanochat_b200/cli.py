"""Command line: generate from a model folder, or replay a trace of token ids.

    python -m nanochat_b200.cli generate --model DIR --tokens 5,17,3 --max-tokens 32 [--temperature T --top-k K]
    python -m nanochat_b200.cli replay --model DIR --dtype bfloat16|float32 --out DIR --max-tokens N < steps

``replay`` reads one JSON object per line, ``{"step": n, "entries": [{"id", "tokens", "want"}], "end": [ids]}``:
the next tokens of each entry's sequence and the places among them whose logits are wanted.  It writes
these to OUT/<step>.f32 (little-endian fp32, rows in the order of the entries and places), then prints
``done <step>``; the sequences in ``end`` give back what they hold.
"""
import argparse
import json
import os
import sys


def _dtype(name):
    import torch
    return {"bfloat16": torch.bfloat16, "float32": torch.float32}[name]


class TokenIds:
    """Stands in for a tokenizer where prompts and answers are token ids: no special tokens."""

    def encode_special(self, s):
        return -1

    def get_bos_token_id(self):
        return -1

    def encode(self, s, prepend=None):
        raise ValueError("this model folder has no tokenizer; use token ids")

    def decode(self, ids):
        return " ".join(str(i) for i in ids)


def replay(args, steps, announce):
    import torch

    from . import ops
    from .engine import SequenceRunner
    from .models import load_model

    model = load_model(args.model, _dtype(args.dtype))
    if getattr(model, "dtype", None) not in (None, _dtype(args.dtype)) or (
            args.dtype == "float32" and not hasattr(model, "dtype")):
        print(f"{type(model).__name__} does not run in {args.dtype}", file=sys.stderr)
        return 3
    runner = SequenceRunner(model, args.max_tokens)
    for line in steps:
        if not line.strip():
            continue
        step = json.loads(line)
        rows = []
        for e in step["entries"]:
            logits = runner.feed(e["id"], e["tokens"], e["want"])
            if logits is not None:
                rows.append(logits)
        if rows:
            out = torch.cat(rows).float().cpu().numpy().astype("<f4")
            ops.check_status(model.get_device())
            path = os.path.join(args.out, f"{step['step']}.f32")
            with open(path + ".part", "wb") as f:
                f.write(out.tobytes())
            os.replace(path + ".part", path)
        for seq_id in step.get("end", []):
            runner.finish(seq_id)
        announce(f"done {step['step']}")
    torch.cuda.synchronize()
    ops.check_status(model.get_device())
    return 0


def generate(args):
    from .engine import Engine
    from .models import load_model

    model = load_model(args.model, _dtype(args.dtype))
    prompt = [int(t) for t in args.tokens.replace(",", " ").split()]
    engine = Engine(model, TokenIds(), page_tokens=args.page_tokens)
    results, _ = engine.generate_batch(prompt, num_samples=args.num_samples, max_tokens=args.max_tokens,
                                       temperature=args.temperature, top_k=args.top_k, seed=args.seed)
    for row in results:
        print(" ".join(str(t) for t in row[len(prompt):]))
    return 0


def main(argv=None):
    ap = argparse.ArgumentParser(prog="nanochat_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue a prompt of token ids")
    r = sub.add_parser("replay", help="feed a trace of token ids and write logits")
    for p in (g, r):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
        p.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
        p.add_argument("--max-tokens", type=int, required=True)
    g.add_argument("--tokens", required=True, help="prompt token ids, separated by commas or spaces")
    g.add_argument("--num-samples", type=int, default=1)
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--top-k", type=int, default=None)
    g.add_argument("--seed", type=int, default=42)
    g.add_argument("--page-tokens", type=int, default=None, help="keep keys and values in pages of this many tokens")
    r.add_argument("--out", required=True, help="existing folder for the logits")
    args = ap.parse_args(argv)
    if args.command == "generate":
        return generate(args)
    return replay(args, sys.stdin, lambda text: print(text, flush=True))


if __name__ == "__main__":
    sys.exit(main())
