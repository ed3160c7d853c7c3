"""Generation from the command line, on token ids.

    python -m teenygrad_b200.generate --model DIR --prompt 5,17,3 [--prompt 8,1 ...] --max-new-tokens 32
                                      [--dtype float32] [--temperature 0.8 --top-k 50 --top-p 0.95 --seed 1]

DIR holds config.json and model.safetensors; the model class follows from the configuration.  Prints one line of new token
ids per prompt.
"""
import argparse

import torch

DTYPES = {"bfloat16": torch.bfloat16, "float32": torch.float32}


def parse_args(argv=None):
    p = argparse.ArgumentParser(prog="python -m teenygrad_b200.generate", description=__doc__.split("\n")[0])
    p.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    p.add_argument("--prompt", action="append", required=True, help="comma-separated token ids; repeat for a batch")
    p.add_argument("--max-new-tokens", type=int, default=32)
    p.add_argument("--dtype", choices=sorted(DTYPES), default="bfloat16")
    p.add_argument("--temperature", type=float, default=0.0, help="0 = greedy")
    p.add_argument("--top-k", type=int, default=50)
    p.add_argument("--top-p", type=float, default=1.0)
    p.add_argument("--seed", type=int, default=0)
    p.add_argument("--no-graph", action="store_true", help="launch the decode kernels one by one")
    args = p.parse_args(argv)
    args.prompt = [[int(t) for t in s.split(",")] for s in args.prompt]
    return args


def main(argv=None):
    args = parse_args(argv)
    from . import models
    n, longest = len(args.prompt), max(len(p) for p in args.prompt)
    model = models.load(args.model, DTYPES[args.dtype], max_batch=n, max_len=longest + args.max_new_tokens,
                        max_new_tokens=args.max_new_tokens)
    model.set_sampling(args.temperature, args.top_k, args.top_p, args.seed)
    prompts = torch.tensor(args.prompt) if all(len(p) == longest for p in args.prompt) else args.prompt
    for row in model.generate(prompts, args.max_new_tokens, use_graph=not args.no_graph).tolist():
        print(",".join(map(str, row)))


if __name__ == "__main__":
    main()
