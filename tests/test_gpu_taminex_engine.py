"""The Taminex family through the engine — scheduler, cache pools, state slots, captured graphs, sampler, command line —
against the plain CPU restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import taminex_fixtures as fx
from engine_helpers import agree, error, make_engine, portions, run, write_model
from oracle import taminex as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 6e-5, torch.bfloat16: 4e-2}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer(dtype, monkeypatch):
    from llm_from_scratch_b200 import ops
    cfg = fx.config()
    w, ids, want, got = fx.weights(cfg, 1), fx.tokens(cfg, 90, 3), [], []
    orc.forward(cfg, w, ids, collect=want)
    plain = ops.residual_norm

    def spy(x, *a, **k):
        h = plain(x, *a, **k)
        got.append(x[:90].double().cpu())
        return h

    eng = make_engine(cfg, w, dtype)
    monkeypatch.setattr(ops, "residual_norm", spy)
    run(eng, portions(ids, [90]))
    at = np.cumsum([1 + (l["mlp"] is not None) for l in cfg["layers"]])
    assert len(got) == at[-1] + 1
    for i, x in zip(at, want):
        assert ((got[i] - x).pow(2).mean().sqrt() / x.std()).item() < TOL[dtype], i
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_portions_and_single_tokens_give_the_same_logits(dtype):
    cfg = fx.config()
    w = fx.weights(cfg, 1)
    eng = make_engine(cfg, w, dtype)
    assert eng.model_runner.graphs          # single tokens replay captured graphs
    for n, sizes_list in ((150, [[150], [1], [2], [3, 1, 16], [64, 7, 2, 33]]), (1, [[1]]), (3, [[3], [2, 1], [1]]),
                          (17, [[16, 1], [17]])):
        ids = fx.tokens(cfg, n, n)
        want = orc.forward(cfg, w, ids)
        for sizes in sizes_list:
            assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[dtype], sizes
    eng.exit()


VARIANTS = {
    "ones": fx.config([fx.delta(heads=1, kv_heads=1, dim=16, vdim=16, conv=1, ff=8), fx.latent(heads=1, dim=16, vdim=16, kv_rank=16,
                                                                                           ff=8),
                       fx.attention(heads=1, kv_heads=1, dim=16, vdim=16, dims=2, ff=8)], vocab=17, width=24),
    "odd": fx.config([fx.delta(heads=3, kv_heads=1, dim=10, vdim=6, conv=3, ff=30), fx.attention(heads=3, kv_heads=3, dim=18, vdim=11,
                                                                                            dims=18, ff=None),
                      fx.latent(heads=3, dim=7, vdim=9, kv_rank=21), fx.latent(heads=2, dim=5, vdim=3, kv_rank=21, kv_from=2, ff=None)],
                     vocab=101, width=50, eps=1e-3, cap=3.0),
    "wide": fx.config([fx.attention(heads=8, kv_heads=2, dim=64, vdim=64, dims=64, ff=256, base=1e6),
                       fx.delta(heads=4, kv_heads=2, dim=128, vdim=128, ff=96), fx.latent(heads=16, dim=64, vdim=64, kv_rank=256),
                       fx.attention(heads=4, kv_heads=2, dim=128, vdim=128, dims=32), fx.latent(heads=4, dim=128, vdim=128,
                                                                                             kv_rank=256, kv_from=2),
                       fx.delta(heads=2, kv_heads=2, dim=64, vdim=64)], vocab=260, width=256, scale=0.4),
    "only delta": fx.config([fx.delta(), fx.delta(heads=2, kv_heads=1, dim=48, vdim=16, conv=2)]),
    "no state": fx.config([fx.latent(), fx.attention(dims=0), fx.latent(kv_from=0)], cap=25.0),
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


KINDS = {"attention": [fx.attention(heads=4, kv_heads=2, dim=64, vdim=64, dims=32)],
         "latent": [fx.latent(heads=4, dim=32, vdim=32), fx.delta()],
         "shared": [fx.latent(heads=2, dim=32, vdim=32, ff=None), fx.delta(), fx.latent(heads=4, dim=32, vdim=32, kv_from=0)]}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(KINDS))
def test_a_marked_key_counts_wherever_it_is(kind, dtype):
    """One earlier token that stands out: the first of the sequence, beside page borders, inside the same portion, in an
    earlier one, and far back, for queries inside a prompt and for decoded ones."""
    cfg = fx.config(KINDS[kind], cap=30.0)
    w = fx.marked_keys(cfg, fx.weights(cfg, 4))
    n = 330
    base = fx.plain_tokens(cfg, n, 8)
    eng = make_engine(cfg, w, dtype)
    for last in (n - 1, 257, 256, 255):
        for at in (0, 1, 15, 16, 63, 64, last - 1, last - 17):
            ids = list(base)
            ids[last] = fx.SEEK
            alone = orc.forward(cfg, w, ids[:last + 1])[last]
            ids[at] = fx.MARK
            want = orc.forward(cfg, w, ids[:last + 1])
            effect = ((want[last] - alone).pow(2).mean().sqrt() / want.std()).item()
            assert effect > 4 * TOL[torch.bfloat16], (last, at, effect)
            for sizes in ([n], [last, 1], [last - 1, 2], [at + 1, 2, n]):
                got = run(eng, portions(ids[:last + 1], sizes))["a"]
                assert error(got[last:], want[last:]) < TOL[dtype], (last, at, sizes)
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


@pytest.mark.parametrize("dtype", DTYPES)
def test_a_request_does_not_see_its_neighbours(dtype):
    """The same request alone and beside others, in the same portions: equal up to rounding in the last bits."""
    cfg = fx.config()
    w = fx.weights(cfg, 6)
    a, b, c = (fx.tokens(cfg, n, n) for n in (75, 60, 90))
    eng = make_engine(cfg, w, dtype)
    alone = run(eng, portions(a, [40, 1, 2, 32]))["a"]
    at = [0, 40, 41, 43, 75]
    steps = [([("b", b[i * 15:(i + 1) * 15]), ("a", a[at[i]:at[i + 1]]), ("c", c[i:i + 1])], ["a", "b", "c"] if i == 3 else [])
             for i in range(4)]
    beside = run(eng, steps)["a"]
    assert error(beside, alone.double()) < (1e-5 if dtype == torch.float32 else 2e-2)
    eng.exit()


@pytest.mark.parametrize("dtype,slack", [(torch.float32, 3e-4), (torch.bfloat16, 0.12)])
@pytest.mark.parametrize("kw", [dict(), dict(max_num_batched_tokens=64), dict(enforce_eager=True), dict(decode_window=5),
                                dict(max_num_batched_tokens=24), dict(max_num_batched_tokens=40, max_cached_blocks=11)])
def test_greedy_generation_through_the_scheduler(kw, dtype, slack):
    """``LLMEngine.generate``: more requests than slots; with a small budget prompts are read in portions beside
    decoding sequences; with a small pool sequences are preempted and recomputed."""
    from llm_from_scratch_b200.engine import SamplingParams
    cfg = fx.config()
    w = fx.weights(cfg, 7)
    prompts = [fx.tokens(cfg, n, 90 + n) for n in (40, 3, 77, 16, 1, 33, 50)]
    eng = make_engine(cfg, w, dtype, max_tokens=1024, **{"max_num_batched_tokens": 512, **kw})
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


def test_greedy_with_a_negative_logit_scale():
    from llm_from_scratch_b200.engine import SamplingParams
    cfg = fx.config([fx.delta(), fx.attention()], scale=-0.8)
    w = fx.weights(cfg, 7)
    prompts = [fx.tokens(cfg, 20, 1)]
    eng = make_engine(cfg, w, torch.float32)
    out = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=12, ignore_eos=True))["token_ids"]
    agree(orc, out, cfg, w, prompts, 3e-4)
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
