"""The Meresun family through the engine — scheduler, cache pools, captured graphs, sampler, command line — against the plain
CPU restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import meresun_fixtures as fx
from engine_helpers import agree, make_engine, portions, run, write_model
from meresun_fixtures import error, reference
from oracle import meresun as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 6e-5, torch.bfloat16: 3e-2}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer_run(dtype, monkeypatch):
    from llm_from_scratch_b200 import ops
    cfg = fx.config()
    w, ids, want, got = fx.weights(cfg, 1), fx.tokens(cfg, 90, 3), [], []
    orc.forward(cfg, w, ids, collect=want)
    settled = reference(cfg, w, ids, dtype)[1]
    start = w["embed"][ids].double() * cfg["embedding"]["scale"]
    again = [a for _, a in orc.layer_runs(cfg)] + [False]
    plain = ops.residual_group_norm

    def spy(x, *a, **k):
        h = plain(x, *a, **k)
        got.append(x[:90].double().cpu())
        return h

    eng = make_engine(cfg, w, dtype)
    monkeypatch.setattr(ops, "residual_group_norm", spy)
    run(eng, portions(ids, [90]))
    assert len(got) == len(want) + 1
    for i, x in enumerate(want):
        x = x + start if again[i + 1] else x
        assert ((got[i + 1] - x)[settled].pow(2).mean(-1).sqrt().max() / x.std()).item() < TOL[dtype], i
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_portions_and_single_tokens_give_the_same_logits(dtype):
    cfg = fx.config()
    w = fx.weights(cfg, 1)
    eng = make_engine(cfg, w, dtype)
    assert eng.model_runner.graphs          # single tokens replay captured graphs
    for n, sizes_list in ((150, [[150], [1], [2], [3, 1, 16], [64, 7, 2, 33], [37, 36, 38]]), (1, [[1]]), (3, [[3], [2, 1], [1]]),
                          (17, [[16, 1], [17]])):
        ids = fx.tokens(cfg, n, n)
        want = reference(cfg, w, ids, dtype)
        for sizes in sizes_list:
            assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[dtype], sizes
    eng.exit()


def test_portions_gather_only_what_their_windows_reach(monkeypatch):
    from llm_from_scratch_b200 import ops
    cfg = fx.config([fx.layer(fx.dense(), window=20), fx.layer(fx.dense(), window=0), fx.layer(fx.dense(), window=90)], loop=None)
    w, ids = fx.weights(cfg, 1), fx.tokens(cfg, 120, 3)
    want, totals = reference(cfg, w, ids, torch.float32), []
    plain = ops.gather_rows
    monkeypatch.setattr(ops, "gather_rows", lambda *a, **k: (totals.append(a[4]), plain(*a, **k))[1])
    eng = make_engine(cfg, w, torch.float32)
    assert error(run(eng, portions(ids, [60, 10, 50]))["a"], want) < TOL[torch.float32]
    assert totals == [29, 70, 70, 69, 120, 120]
    eng.exit()


VARIANTS = {
    "ones": fx.config([fx.layer(fx.moe(ff=8, experts=1, top=1, groups=(1, 1)), heads=1, dim=8, rot_dim=8, vdim=8, q_rank=8, kv_rank=8,
                                window=1)], vocab=17, width=24, groups=1, side=5, loop=None),
    "odd": fx.config([fx.layer(fx.moe(ff=21, experts=6, top=1, groups=(6, 2)), heads=3, dim=7, rot_dim=6, vdim=9, q_rank=11, kv_rank=21,
                               window=5),
                      fx.layer(fx.dense(30), heads=2, dim=5, rot_dim=2, vdim=11, q_rank=33, kv_rank=10, window=90, base=30.0)],
                     vocab=101, width=50, eps=1e-3, groups=5, side=29, loop=(0, 2, 3)),
    "wide": fx.config([fx.layer(fx.moe(ff=64, experts=16, top=4, groups=(4, 2)), heads=4, dim=128, rot_dim=64, vdim=128, q_rank=96,
                                kv_rank=512, window=70),
                       fx.layer(fx.dense(512), heads=18, dim=64, rot_dim=16, vdim=72, q_rank=64, kv_rank=256, window=64),
                       fx.layer(fx.dense(256), heads=2, dim=128, rot_dim=64, vdim=128, q_rank=96, kv_rank=256, window=33)],
                      vocab=260, width=256, groups=2, side=32, loop=(0, 1, 2)),
    "no window": fx.config([fx.layer(fx.dense(), window=0), fx.layer(None, window=0, scaling=None, rot_dim=2)], loop=(1, 2, 2)),
    "one layer five times": fx.config([fx.layer(fx.moe(limit=2.5))], groups=1, loop=(0, 1, 5), embed_scale=2.0),
    "unlike layers": fx.config([fx.layer(None, heads=1), fx.layer(fx.dense(16), kv_rank=128, vdim=16, window=200),
                                fx.layer(fx.moe(experts=40, top=6, groups=(4, 3))), fx.layer(fx.dense(200), q_rank=200)], loop=(3, 4, 2)),
}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", sorted(VARIANTS))
def test_other_sizes(name, dtype):
    cfg = VARIANTS[name]
    w = fx.weights(cfg, 2)
    ids = fx.tokens(cfg, 140, 5)
    want = reference(cfg, w, ids, dtype)
    eng = make_engine(cfg, w, dtype, block_size=64)
    for sizes in ([140], [100, 2, 1, 30, 1]):
        assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[dtype]
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_on_pages_that_are_used_again(dtype):
    """Portions beside single tokens, requests left out of steps, twelve requests over a pool that holds little more than
    the four live ones: every request's logits equal its logits alone."""
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
        assert error(got[name], reference(cfg, w, ids[name], dtype)) < TOL[dtype], name
    assert eng.scheduler.block_manager.num_free_blocks == eng.model_runner.num_kv_blocks
    eng.exit()


KINDS = {"narrow": fx.config([fx.layer(fx.dense(), heads=4, window=48)], loop=None, groups=1),
         "page": fx.config([fx.layer(fx.moe(), heads=2, window=64)], loop=None),
         "tensor cores": fx.config([fx.layer(fx.dense(), heads=2, dim=128, rot_dim=64, vdim=128, kv_rank=256, window=100)], loop=None),
         "whole": fx.config([fx.layer(fx.dense(), window=0)], loop=None),
         "loop": fx.config([fx.layer(fx.dense(), window=48), fx.layer(fx.dense(), window=48)], loop=(0, 1, 2))}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(KINDS))
def test_a_marked_key_counts_inside_the_window_only(kind, dtype):
    """One earlier token that stands out: just inside and just outside the window, beside page borders, inside the same
    portion and in an earlier one, the first of the sequence, far back; for queries inside a prompt and for decoded ones.
    A layer alone does not notice the token outside its window; layers behind one another do."""
    cfg = KINDS[kind]
    w = fx.marked_keys(cfg, fx.weights(cfg, 4))
    n, window = 330, cfg["layers"][0]["mixer"]["mask"]["size"] if cfg["layers"][0]["mixer"]["mask"] else 0
    base = fx.plain_tokens(cfg, n, 8)
    eng = make_engine(cfg, w, dtype)
    seen = 0
    for last in (n - 1, 257, 256, 40):
        alone = orc.forward(cfg, w, base[:last] + [fx.SEEK])[last]
        for at in sorted({0, 15, 16, 64, last - 1, last - 17, last - window, last - window + 1} & set(range(last))):
            ids = list(base[:last]) + [fx.SEEK]
            ids[at] = fx.MARK
            want, settled = reference(cfg, w, ids, dtype)
            effect = ((want[last] - alone).pow(2).mean().sqrt() / want.std()).item()
            if window == 0 or last - at < window:
                assert effect > 4 * TOL[torch.bfloat16], (last, at, effect)
                seen += 1
            elif len(orc.layer_runs(cfg)) == 1:
                assert effect == 0.0
            for sizes in ([n], [last, 1], [last - 1, 2], [at + 1, 2, n]):
                got = run(eng, portions(ids, sizes))["a"]
                assert error(got[last:], (want[last:], settled[last:])) < TOL[dtype], (last, at, sizes)
    assert seen >= 6
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_behind_a_short_prompt(dtype):
    cfg = fx.config()
    w = fx.weights(cfg, 6)
    ids = fx.tokens(cfg, 330, 9)
    want = reference(cfg, w, ids, dtype)
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
    settled = reference(cfg, w, a, dtype)[1]
    assert error(beside, (alone.double(), settled)) < (1e-5 if dtype == torch.float32 else 2e-2)
    eng.exit()


@pytest.mark.parametrize("dtype,slack", [(torch.float32, 3e-4), (torch.bfloat16, 0.15)])
@pytest.mark.parametrize("kw", [dict(), dict(max_num_batched_tokens=64), dict(enforce_eager=True), dict(decode_window=5),
                                dict(max_num_batched_tokens=24), dict(max_num_batched_tokens=40, max_cached_blocks=11)])
def test_greedy_generation_through_the_scheduler(kw, dtype, slack):
    """``LLMEngine.generate``: more requests than places; with a small budget prompts are read in portions beside decoding
    sequences; with a small pool sequences are preempted and recomputed."""
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
    eng.exit()


@pytest.mark.parametrize("dtype,slack", [(torch.float32, 3e-4), (torch.bfloat16, 0.15)])
def test_captured_steps_of_whole_prompts(dtype, slack):
    """Steps of new prompts replay a graph in bf16 (padded batches of unlike lengths, windows, experts); steps with single
    tokens or with the rest of a prompt do not.  The general fp32 kernels are never captured."""
    from llm_from_scratch_b200.engine import SamplingParams
    cfg = fx.config()
    w = fx.weights(cfg, 7)
    prompts = [fx.tokens(cfg, n, 90 + n) for n in (40, 3, 77, 130, 2, 33, 50, 200)]
    eng = make_engine(cfg, w, dtype, max_tokens=2048, max_num_batched_tokens=256, prefill_graphs=True)
    runner, replayed = eng.model_runner, []
    original = runner._replay_prefill
    runner._replay_prefill = lambda seqs: (lambda h: (replayed.append(h is not None), h)[1])(original(seqs))
    out = eng.generate(prompts, SamplingParams(temperature=0.0, max_tokens=13, ignore_eos=True))["token_ids"]
    agree(orc, out, cfg, w, prompts, slack)
    assert bool(runner.prefill_graphs) == (dtype == torch.bfloat16)
    if dtype == torch.bfloat16:
        assert True in replayed and False in replayed
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


def test_a_prompt_large_enough_for_the_compute_bound_expert_kernels():
    """Hundreds of rows per expert: the 256-row grouped GEMM, and above its limit the library's."""
    from llm_from_scratch_b200.model.mixers import GroupedMoE
    cfg = fx.config([fx.layer(fx.moe(ff=64, experts=4, top=2, groups=(2, 1)))], width=128, groups=2, loop=None)
    w = fx.weights(cfg, 5)
    ids = fx.tokens(cfg, 700, 1)
    want = reference(cfg, w, ids, torch.bfloat16)
    for limit in (GroupedMoE.own_gemm_max_rows_per_expert, 1 << 20):
        eng = make_engine(cfg, w, torch.bfloat16, max_tokens=1024)
        eng.model_runner.model.layers[0].sublayers.mlp.own_gemm_max_rows_per_expert = limit
        assert error(run(eng, portions(ids, [700]))["a"], want) < TOL[torch.bfloat16]
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
    (la, ka), (lb, kb) = (reference(cfg, w, ids, getattr(torch, dtype)) for ids in (a, b))
    pick = lambda x, y: {0: x[[0, 17]], 1: torch.stack([y[65], y[3], x[18]]), 3: torch.stack([x[19], y[69]])}
    want, settled = pick(la, lb), pick(ka, kb)
    assert not os.path.exists(tmp_path / "2.f32")
    for i, x in want.items():
        got = torch.from_numpy(np.fromfile(tmp_path / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]).copy())
        assert error(got, (x, settled[i])) < TOL[getattr(torch, dtype)]


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
