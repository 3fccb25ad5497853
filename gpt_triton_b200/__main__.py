"""Command line:

    python -m gpt_triton_b200 info --model DIR
    python -m gpt_triton_b200 generate --model DIR --ids 5,17,3 [--ids ...] --new-tokens 32 [--temperature T --top-k K --seed S]

Token ids in, token ids out (the package has no tokenizer).  Prompts of equal length run as one batch.
"""

import argparse
import sys


def main(argv=None):
    ap = argparse.ArgumentParser(prog="python -m gpt_triton_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    info = sub.add_parser("info", help="architecture and size of a model folder")
    gen = sub.add_parser("generate", help="continue prompts given as token ids")
    for p in (info, gen):
        p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    gen.add_argument("--ids", action="append", required=True, metavar="ID,ID,...", help="a prompt; may be repeated")
    gen.add_argument("--new-tokens", type=int, default=16)
    gen.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float16", "float32"])
    gen.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    gen.add_argument("--top-k", type=int, default=0, help="0 = all")
    gen.add_argument("--seed", type=int, default=0)
    gen.add_argument("--portion", type=int, default=0, help="run prompts in pieces of at most this many tokens (0 = whole)")
    args = ap.parse_args(argv)

    from .checkpoint import read_config
    from .registry import architecture_of

    if args.command == "info":
        import os

        from .checkpoint import read_safetensors

        tensors = read_safetensors(os.path.join(args.model, "model.safetensors"))
        print(f"{architecture_of(read_config(args.model))}: {len(tensors)} tensors, {sum(t.numel() for t in tensors.values())} parameters")
        return 0

    import torch

    from .build import build

    build()
    from .registry import load_model

    prompts = [[int(t) for t in text.split(",")] for text in args.ids]
    model = load_model(args.model, dtype=getattr(torch, args.dtype))
    results = [None] * len(prompts)
    for length in sorted({len(p) for p in prompts}):
        group = [i for i, p in enumerate(prompts) if len(p) == length]
        ids = torch.tensor([prompts[i] for i in group], device="cuda")
        out = model.generate(ids, args.new_tokens, temperature=args.temperature, top_k=args.top_k, seed=args.seed, portion=args.portion)
        for i, row in zip(group, out.tolist()):
            results[i] = row
    for row in results:
        print(",".join(map(str, row)))
    return 0


if __name__ == "__main__":
    sys.exit(main())
