"""The Nabalix family through the engine — scheduler, cache pools, state slots, captured graphs, sampler, command
line — against the plain CPU restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import nabalix_fixtures as fx
from engine_helpers import agree, error, make_engine, portions, run, write_model
from oracle import nabalix as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 6e-5, torch.bfloat16: 4e-2}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_portions_and_single_tokens_give_the_same_logits(dtype):
    cfg = fx.config()
    w = fx.weights(cfg, 1)
    eng = make_engine(cfg, w, dtype)
    assert eng.model_runner.graphs          # single tokens replay captured graphs
    for n, sizes_list in ((150, [[150], [1], [2], [3, 1, 16], [64, 7, 2, 33]]), (1, [[1]]), (17, [[16, 1], [17]])):
        ids = fx.tokens(cfg, n, n)
        want = orc.forward(cfg, w, ids)
        for sizes in sizes_list:
            got = run(eng, portions(ids, sizes))["a"]
            assert error(got, want) < TOL[dtype], sizes
    eng.exit()


VARIANTS = {
    "ones": fx.config([fx.layer(heads=1, kv_heads=1, dim=16, vdim=16, window=1, rec=(1, 16, 16), ff=8)], vocab=17, width=24,
                      streams=1),
    "odd": fx.config([fx.layer(heads=3, kv_heads=3, dim=12, vdim=20, window=5, rec=(2, 10, 6), ff=30), fx.layer(
        heads=3, kv_heads=1, dim=20, vdim=12, window=300, rec=(1, 30, 7), ff=None)], vocab=101, width=50, streams=5, eps=1e-3),
    "wide": fx.config([fx.layer(heads=16, kv_heads=4, dim=64, vdim=64, window=48, rec=(2, 128, 64), ff=256),
                       fx.layer(heads=24, kv_heads=2, dim=32, vdim=128, window=65, rec=(4, 64, 128), ff=96, softcap=3.0)],
                      vocab=260, width=256, streams=4),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(VARIANTS))
def test_other_sizes(name, dtype):
    cfg = VARIANTS[name]
    w = fx.weights(cfg, 2)
    ids = fx.tokens(cfg, 140, 5)
    want = orc.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype, block_size=64)
    for sizes in ([140], [100, 2, 1, 30, 1]):
        assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[dtype] * (2 if name == "ones" else 1)
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_on_pages_and_slots_that_are_used_again(dtype):
    """Portions beside single tokens, requests left out of steps, twelve requests over four slots and a pool that
    holds little more than the live ones: every request's logits equal its logits alone."""
    cfg = fx.config()
    w = fx.weights(cfg, 3)
    rng = np.random.default_rng(0)
    lens = [int(x) for x in rng.integers(1, 130, 12)]
    ids = {f"r{i}": fx.tokens(cfg, n, 50 + i) for i, n in enumerate(lens)}
    eng = make_engine(cfg, w, dtype, max_tokens=4 * 144)
    todo, live, steps = list(ids), {}, []
    while todo or live:
        while todo and len(live) < 4:
            live[todo.pop(0)] = 0
        entries, end = [], []
        for name in list(live):
            if rng.random() < 0.25 and len(live) > 1:
                continue
            n = int(rng.choice([1, 1, 1, 2, 3, 16, 29, 64]))
            part = ids[name][live[name]:live[name] + n]
            entries.append((name, part))
            live[name] += len(part)
            if live[name] == len(ids[name]):
                end.append(name)
                del live[name]
        if entries:
            steps.append((entries, end))
    got = run(eng, steps)
    for name in ids:
        assert error(got[name], orc.forward(cfg, w, ids[name])) < TOL[dtype], name
    assert eng.scheduler.block_manager.num_free_blocks == eng.model_runner.num_kv_blocks
    assert len(eng.scheduler.state_slots.free) == 4
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("window", [16, 33])
def test_a_marked_key_counts_up_to_the_window_edge_and_not_beyond(window, dtype):
    """One earlier token that stands out, at the last distance the window holds, at the first it does not, and at
    page borders, for queries inside a prompt and for decoded ones."""
    cfg = fx.config([fx.layer(window=window, softcap=50.0)], streams=2)
    w = fx.marked_keys(cfg, fx.weights(cfg, 4))
    n = 100
    base = fx.plain_tokens(cfg, n, 8)
    eng = make_engine(cfg, w, dtype)
    seen_effect = {}
    for last in (n - 1, 63, 64):
        for back in (window - 1, window, 15, 1):
            ids = list(base)
            ids[last], ids[last - back] = fx.SEEK, fx.MARK
            want = orc.forward(cfg, w, ids)
            for sizes in ([n], [last, 1, n], [last - 1, 2, n], [last - back, 1, 1, 1, n]):
                got = run(eng, portions(ids, sizes))["a"]
                assert error(got, want) < TOL[dtype], (last, back, sizes)
            ids[last - back] = base[last - back]
            alone = orc.forward(cfg, w, ids)[last]
            seen_effect[back] = ((want[last] - alone).pow(2).mean().sqrt() / want.std()).item()
    # the mark decides the logits inside the window only (what is left outside runs through the recurrence)
    assert seen_effect[window - 1] > 5 * TOL[torch.bfloat16]
    assert seen_effect[window - 1] > 1.5 * seen_effect[window]
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_behind_a_short_prompt(dtype):
    cfg = fx.config()
    w = fx.weights(cfg, 6)
    ids = fx.tokens(cfg, 330, 9)
    want = orc.forward(cfg, w, ids)
    eng = make_engine(cfg, w, dtype, block_size=64)
    assert error(run(eng, portions(ids, [5] + [1] * 325))["a"], want) < TOL[dtype]
    eng.exit()


@pytest.mark.parametrize("dtype,slack", [(torch.float32, 3e-4), (torch.bfloat16, 0.12)])
@pytest.mark.parametrize("kw", [dict(), dict(prefill_graphs=True), dict(prefill_graphs=True, max_num_batched_tokens=64),
                                dict(enforce_eager=True), dict(decode_window=5), dict(max_num_batched_tokens=24),
                                dict(max_num_batched_tokens=40, max_cached_blocks=11)])
def test_greedy_generation_through_the_scheduler(kw, dtype, slack):
    """``LLMEngine.generate``: more requests than slots; with a small budget prompts are read in portions beside
    decoding sequences; with a small pool sequences are preempted and recomputed."""
    from llm_from_scratch_b200.engine import SamplingParams
    cfg = fx.config()
    w = fx.weights(cfg, 7)
    prompts = [fx.tokens(cfg, n, 90 + n) for n in (40, 3, 77, 16, 1, 33, 50)]
    eng = make_engine(cfg, w, dtype, max_tokens=1024, max_num_batched_tokens=kw.pop("max_num_batched_tokens", 512), **kw)
    assert bool(eng.model_runner.prefill_graphs) == ("prefill_graphs" in kw and dtype == torch.bfloat16)
    preempted = []
    original = eng.scheduler.preempt
    eng.scheduler.preempt = lambda s: (preempted.append(s), original(s))
    out = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=25, ignore_eos=True))["token_ids"]
    assert [len(t) for t in out] == [24] * len(prompts)
    agree(orc, out, cfg, w, prompts, slack)
    assert bool(preempted) == ("max_cached_blocks" in kw)
    assert eng.scheduler.block_manager.num_free_blocks == eng.model_runner.num_kv_blocks
    assert len(eng.scheduler.state_slots.free) == 4
    eng.exit()


def test_sampling_with_temperature_and_an_end_token():
    from llm_from_scratch_b200.engine import SamplingParams
    cfg = fx.config()
    w = fx.weights(cfg, 7)
    eng = make_engine(cfg, w, torch.bfloat16)
    prompts = [fx.tokens(cfg, 9, 1), fx.tokens(cfg, 30, 2)]
    a = eng.generate(prompts, SamplingParams(temperature=1.0, max_tokens=20, ignore_eos=True))["token_ids"]
    assert all(0 <= t < cfg["vocab"] for s in a for t in s) and len(set(a[0] + a[1])) > 5
    eng.scheduler.eos = first = eng.generate([prompts[0]], SamplingParams(temperature=0.0, max_tokens=4))["token_ids"][0][0]
    assert eng.generate([prompts[0]], SamplingParams(temperature=0.0, max_tokens=20))["token_ids"][0] == [first]
    eng.exit()


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_trace_command_line(dtype, tmp_path):
    cfg = fx.config()
    w = fx.weights(cfg, 11)
    write_model(tmp_path / "m", cfg, w)
    a, b = fx.tokens(cfg, 20, 1), fx.tokens(cfg, 70, 2)
    steps = [dict(step=0, entries=[dict(id="a", tokens=a[:18], want=[0, 17])], end=[]),
             dict(step=1, entries=[dict(id="b", tokens=b[:66], want=[65, 3]), dict(id="a", tokens=a[18:19], want=[0])], end=[]),
             dict(step=2, entries=[dict(id="b", tokens=b[66:69], want=[])], end=[]),
             dict(step=3, entries=[dict(id="a", tokens=a[19:], want=[0]), dict(id="b", tokens=b[69:], want=[0])], end=["a", "b"])]
    r = subprocess.run([os.path.join(ROOT, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out",
                        str(tmp_path), "--max-tokens", "192"], input="".join(json.dumps(s) + "\n" for s in steps),
                       capture_output=True, text=True, timeout=300)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.splitlines() if x.startswith("done")] == [f"done {i}" for i in range(4)]
    la, lb = orc.forward(cfg, w, a), orc.forward(cfg, w, b)
    want = {0: la[[0, 17]], 1: torch.stack([lb[65], lb[3], la[18]]), 3: torch.stack([la[19], lb[69]])}
    assert not os.path.exists(tmp_path / "2.f32")
    for i, x in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
        assert error(got, x) < TOL[getattr(torch, dtype)]


def test_generate_command_line(tmp_path):
    cfg = fx.config()
    w = fx.weights(cfg, 11)
    write_model(tmp_path / "m", cfg, w)
    prompts = [fx.tokens(cfg, 12, 1), fx.tokens(cfg, 5, 2)]
    r = subprocess.run([sys.executable, "-m", "llm_from_scratch_b200", "generate", "--model", str(tmp_path / "m"), "--dtype",
                        "float32", "--max-tokens", "9", "--ignore-eos"] + [" ".join(map(str, p)) for p in prompts],
                       capture_output=True, text=True, timeout=300, cwd=ROOT)
    assert r.returncode == 0, r.stderr[-2000:]
    agree(orc, [json.loads(x)["token_ids"] for x in r.stdout.splitlines()], cfg, w, prompts, 3e-4)
