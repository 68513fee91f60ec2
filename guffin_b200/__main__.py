"""Command line: `python -m guffin_b200 models | info | generate`.

There is no tokenizer in this package: prompts and generated text are token ids.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def _prompts(args) -> list:
    prompts = [[int(t) for t in text.replace(",", " ").split()] for text in args.tokens or []]
    if args.tokens_file:
        with (sys.stdin if args.tokens_file == "-" else open(args.tokens_file)) as f:
            prompts += [[int(t) for t in line.replace(",", " ").split()] for line in f if line.strip()]
    if not prompts or not all(prompts):
        raise SystemExit("generate needs at least one prompt (--tokens or --tokens-file), each with at least one token id")
    return prompts


def generate(args) -> None:
    from . import engine, model
    prompts = _prompts(args)
    context = args.context or max(len(p) for p in prompts) + args.max_tokens + 1
    options = engine.sampler_options(args.temperature, args.top_k, args.top_p, args.min_p, args.repetition_penalty, args.seed)
    plan = model.Model.open(args.model, context, row_capacity=args.rows, precision=args.dtype)
    if len(prompts) == 1 or args.draft:
        draft = model.Model.open(args.draft, context, row_capacity=2, precision=args.dtype) if args.draft else None
        for prompt in prompts:
            h1 = engine.H1(plan, draft, engine.H1Options(options, int(draft is not None), 0, 0.0, 0, 0))
            h1.prefill(prompt)
            print(" ".join(str(t) for t in h1.generate(args.max_tokens)), flush=True)
    else:
        for row in engine.Batch(plan, prompts, options).generate(args.max_tokens):
            print(" ".join(str(t) for t in row), flush=True)


def info(args) -> None:
    with open(os.path.join(args.model, "config.json")) as f:
        config = json.load(f)
    layers = config["layers"]
    print(f"architecture {config['architecture']}")
    print(f"vocab {config['vocab']}")
    if isinstance(layers, list):
        print(f"width {config['width']}, {len(layers)} layers")
        for i, layer in enumerate(layers):
            mlp = layer.get("mlp") or {"kind": "none"}
            shared = f"  tensors of layer {layer['weights_of']}" if "weights_of" in layer else ""
            print(f"  {i}: {layer['type']} {json.dumps(layer['mixer'])}  {mlp['kind']} {json.dumps({k: v for k, v in mlp.items() if k != 'kind'})}{shared}")
    else:
        print(json.dumps({k: v for k, v in config.items() if k not in ("architecture", "vocab")}))


def main(argv=None) -> int:
    parser = argparse.ArgumentParser(prog="guffin_b200", description=__doc__.splitlines()[0])
    commands = parser.add_subparsers(dest="command", required=True)
    commands.add_parser("models", help="list the architectures config.json may name")
    p = commands.add_parser("info", help="describe a model folder")
    p.add_argument("model")
    p = commands.add_parser("generate", help="generate token ids from prompts of token ids")
    p.add_argument("--model", required=True, help="folder with config.json and model.safetensors or model.gguf")
    p.add_argument("--draft", help="folder of a drafter with the same vocabulary: speculative decoding")
    p.add_argument("--tokens", action="append", help="a prompt's token ids, separated by commas or spaces; several prompts are decoded as one batch")
    p.add_argument("--tokens-file", help="one prompt per line (- for standard input)")
    p.add_argument("--max-tokens", type=int, default=32)
    p.add_argument("--context", type=int, default=0, help="positions the cache is sized for (default: what the prompts need)")
    p.add_argument("--rows", type=int, default=8, help="rows of a pass (1-8): streams that share one pass over the weights")
    p.add_argument("--dtype", choices=("bfloat16", "float32"), default="bfloat16")
    p.add_argument("--temperature", type=float, default=0.0)
    p.add_argument("--top-k", type=int, default=40)
    p.add_argument("--top-p", type=float, default=0.95)
    p.add_argument("--min-p", type=float, default=0.05)
    p.add_argument("--repetition-penalty", type=float, default=1.0)
    p.add_argument("--seed", type=int, default=0)
    args = parser.parse_args(argv)
    from . import build
    build.build()
    if args.command == "models":
        from . import model
        print("\n".join(model.architectures()))
    elif args.command == "info":
        info(args)
    else:
        generate(args)
    return 0


if __name__ == "__main__":
    sys.exit(main())
