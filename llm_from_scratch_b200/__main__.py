"""Command line: ``python -m llm_from_scratch_b200 generate --model DIR "1 2 3" ["4 5"]``.

Reads a model folder (``config.json`` and weights; the model family is the configuration's ``architecture``) and
continues prompts of token ids through ``LLMEngine.generate``; prints one JSON line per prompt.
"""
from __future__ import annotations

import argparse
import json
import os
import sys


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="python -m llm_from_scratch_b200")
    sub = ap.add_subparsers(dest="command", required=True)
    g = sub.add_parser("generate", help="continue prompts of token ids")
    g.add_argument("--model", required=True, help="folder with config.json and weights")
    g.add_argument("--dtype", default="bfloat16", choices=["bfloat16", "float32"])
    g.add_argument("--max-tokens", type=int, default=65, help="stop rule of the engine: max_tokens - 1 tokens are generated")
    g.add_argument("--temperature", type=float, default=0.0)
    g.add_argument("--eos", type=int, default=-1)
    g.add_argument("--ignore-eos", action="store_true")
    g.add_argument("--block-size", type=int, default=16)
    g.add_argument("--max-num-sequences", type=int, default=16)
    g.add_argument("--max-num-batched-tokens", type=int, default=2048)
    g.add_argument("--max-cached-blocks", type=int, default=None, help="KV blocks (default: half of the free memory)")
    g.add_argument("--max-model-length", type=int, default=8192)
    g.add_argument("prompts", nargs="+", help="token ids separated by blanks")
    args = ap.parse_args(argv)

    from . import _build
    with open(os.path.join(args.model, "config.json")) as f:
        _build.ensure(json.load(f).get("architecture"))
    from .engine import SamplingParams
    from .engine.llm_engine import LLMEngine
    prompts = [[int(t) for t in p.split()] for p in args.prompts]
    engine = LLMEngine(dict(model=args.model, dtype=args.dtype, block_size=args.block_size, eos=args.eos,
                            max_num_sequences=args.max_num_sequences, max_num_batched_tokens=args.max_num_batched_tokens,
                            max_cached_blocks=args.max_cached_blocks, max_model_length=args.max_model_length,
                            gpu_memory_utilization=0.5))
    out = engine.generate(prompts, SamplingParams(temperature=args.temperature, max_tokens=args.max_tokens,
                                                  ignore_eos=args.ignore_eos))
    for ids in out["token_ids"]:
        print(json.dumps({"token_ids": ids}))
    engine.exit()
    return 0


if __name__ == "__main__":
    sys.exit(main())
