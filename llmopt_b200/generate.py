"""Generates token ids from a model folder (config.json and model.safetensors):

  python -m llmopt_b200.generate --model DIR --prompt 5,17,3 [--prompt 8,1] [--tokens 32] [--batch 4]
         [--temperature 0.8 --top-k 40 --top-p 0.95 --min-p 0.05 --seed 1] [--stop 2] [--dtype bfloat16|float32]

One line of ids per prompt.  Tokenizers are outside this library: prompts and results are ids."""

from __future__ import annotations

import argparse

from .cuda_native import Runtime
from .decode_engine import create_engine
from .model import load_model


def _ids(text: str) -> list:
    return [int(part) for part in text.replace(",", " ").split()]


def main(argv=None) -> None:
    parser = argparse.ArgumentParser(description="generate token ids from a model folder")
    parser.add_argument("--model", required=True, help="folder with config.json and model.safetensors")
    parser.add_argument("--prompt", required=True, action="append", type=_ids, help="token ids, with commas between them")
    parser.add_argument("--tokens", type=int, default=32, help="most tokens to generate after a prompt")
    parser.add_argument("--batch", type=int, default=8, help="most sequences that decode side by side")
    parser.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    parser.add_argument("--temperature", type=float, default=0.0)
    parser.add_argument("--top-k", type=int, default=0)
    parser.add_argument("--top-p", type=float, default=0.0)
    parser.add_argument("--min-p", type=float, default=0.0)
    parser.add_argument("--seed", type=int, default=1)
    parser.add_argument("--stop", type=_ids, default=[], help="ids that end a sequence")
    args = parser.parse_args(argv)
    config, weights = load_model(args.model)
    capacity = max(len(prompt) for prompt in args.prompt) + args.tokens
    engine = create_engine(Runtime(), config, weights, batch=min(args.batch, len(args.prompt)), capacity=capacity, dtype=args.dtype)
    for tokens in engine.generate(args.prompt, args.tokens, temperature=args.temperature, top_k=args.top_k, top_p=args.top_p,
                                  min_p=args.min_p, seed=args.seed, stop=args.stop):
        print(",".join(map(str, tokens)), flush=True)


if __name__ == "__main__":
    main()
