"""Replays a trace of token ids through the engine, step by step, and returns logits instead of sampling.

Every step names the requests it advances with their next tokens; all of them run as one batch through the
engine's scheduler bookkeeping, cache pools and ``ModelRunner`` — the step function that generation uses, minus
the sampler.  ``main`` is the command line behind ``bin/trace_run``: JSON steps on standard input, raw fp32
logits per step in a folder.
"""
from __future__ import annotations

import argparse
import json
import os
import sys

from .llm_engine import LLMEngine
from .sampling_params import SamplingParams
from .sequence import Sequence


class Replay:
    """Feeds requests of an engine whose model takes mixed batches."""

    def __init__(self, engine: LLMEngine):
        if not getattr(engine.model_runner, "mixed_batches", False):
            raise ValueError("replaying needs a model that takes mixed batches")
        self.engine = engine
        self.live: dict[str, Sequence] = {}

    def step(self, entries: list[tuple[str, list[int], list[int]]], end: list[str] = ()):
        """``entries``: (request id, next tokens, places among them whose logits are wanted).  Returns fp32 logits
        [wanted, vocab] on the device, in the order of the entries; ``end`` names requests finished after the step."""
        sched, runner = self.engine.scheduler, self.engine.model_runner
        batch = []
        for rid, tokens, _ in entries:
            if not tokens:
                raise ValueError(f"request {rid!r} brings no tokens")
            if rid not in self.live:
                self.live[rid] = Sequence([], SamplingParams())
            batch.append((self.live[rid], list(tokens)))
        logits = None
        if batch:
            want = {id(self.live[rid]): list(w) for rid, _, w in entries}
            seqs, is_prefill = sched.feed(batch)
            logits = runner.run_wanted(seqs, is_prefill, [want[id(s)] for s in seqs])
            sched.fed(seqs)
            # the scheduler may reorder a batch: back to the order of the entries
            at, first = {}, 0
            for s in seqs:
                at[id(s)] = first
                first += len(want[id(s)])
            order = [at[id(self.live[rid])] + k for rid, _, w in entries for k in range(len(w))]
            logits = logits[order]
        for rid in end:
            if rid in self.live:
                sched.drop(self.live.pop(rid))
        return logits


def engine_config(model_dir: str, dtype: str, max_tokens: int, block_size: int = 64, max_requests: int = 4, **kw) -> dict:
    """Engine configuration whose pools hold ``max_tokens`` tokens of live requests, at most ``max_requests`` of them."""
    cfg = dict(model=model_dir, dtype=dtype, block_size=block_size, max_num_sequences=max_requests,
               max_num_batched_tokens=max_tokens, max_cached_blocks=(max_tokens + block_size - 1) // block_size, eos=-1,
               device="cuda:0", prefill_token_multiple=64, prefill_graphs=False)
    cfg.update(kw)
    return cfg


def main(argv=None) -> int:
    ap = argparse.ArgumentParser(prog="trace_run", description="Replay a trace of token ids through the engine and "
                                 "write the wanted logits of every step.")
    ap.add_argument("--model", required=True, help="folder with config.json and weights")
    ap.add_argument("--dtype", required=True, choices=["bfloat16", "float32"])
    ap.add_argument("--out", required=True, help="folder for <step>.f32 files")
    ap.add_argument("--max-tokens", required=True, type=int, help="most tokens that live requests hold at any time")
    args = ap.parse_args(argv)

    import torch

    from .. import ops
    engine = LLMEngine(engine_config(args.model, args.dtype, args.max_tokens))
    replay = Replay(engine)
    for line in sys.stdin:
        if not line.strip():
            continue
        step = json.loads(line)
        entries = [(str(e["id"]), e["tokens"], e.get("want", [])) for e in step.get("entries", [])]
        logits = replay.step(entries, [str(i) for i in step.get("end", [])])
        if logits is not None and logits.numel():
            path = os.path.join(args.out, f"{step['step']}.f32")
            with open(path, "wb") as f:
                f.write(logits.float().cpu().numpy().astype("<f4").tobytes())
        ops.check_status()
        sys.stdout.write(f"done {step['step']}\n")
        sys.stdout.flush()
    torch.cuda.synchronize()
    engine.exit()
    return 0
