"""Shared by the engine tests of the families that take mixed batches: an engine over small pools, traces of token
ids through it, and the comparison of its logits with a restatement's."""
import itertools
import json
import os

import torch


def make_engine(cfg, w, dtype, max_tokens=512, block_size=16, **kw):
    from llm_from_scratch_b200.engine import Sequence
    from llm_from_scratch_b200.engine.llm_engine import LLMEngine
    from llm_from_scratch_b200.engine.replay import engine_config
    Sequence.counter = itertools.count()
    return LLMEngine(engine_config(cfg, dtype, max_tokens, block_size, weights=w, **kw))


def error(got, want):
    """Worst position: rms over the vocabulary of the centred difference, in units of the logits' own rms."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / want.std()).max().item()


def run(eng, steps):
    """steps: [([(id, tokens)], [ended ids])]; returns {id: logits of every token}."""
    from llm_from_scratch_b200 import ops
    from llm_from_scratch_b200.engine.replay import Replay
    rep, out = Replay(eng), {}
    for entries, end in steps:
        y = rep.step([(i, t, range(len(t))) for i, t in entries], end)
        ops.check_status()
        for (i, t), part in zip(entries, y.split([len(t) for _, t in entries])):
            out.setdefault(i, []).append(part.cpu())
    return {i: torch.cat(v) for i, v in out.items()}


def portions(ids, sizes, name="a"):
    at, steps = 0, []
    for n in itertools.cycle(sizes):
        part = ids[at:at + n]
        if not part:
            break
        steps.append(([(name, part)], []))
        at += n
    steps[-1] = (steps[-1][0], [name])
    return steps


def agree(orc, streams, cfg, w, prompts, slack):
    """Greedy streams follow the restatement wherever its two best logits are further apart than ``slack``."""
    for got, prompt in zip(streams, prompts):
        logits = orc.forward(cfg, w, list(prompt) + got)[len(prompt) - 1:-1]
        chosen = logits.gather(1, torch.tensor(got)[:, None])[:, 0]
        assert (logits.max(-1).values - chosen).max() <= slack * logits.std(), (logits.max(-1).values - chosen).max()


def write_model(folder, cfg, w):
    from safetensors.torch import save_file
    os.makedirs(folder, exist_ok=True)
    with open(os.path.join(folder, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file({k: v.contiguous() for k, v in w.items()}, os.path.join(folder, "model.safetensors"))
