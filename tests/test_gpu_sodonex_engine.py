"""The Sodonex family through the engine — scheduler, cache pools, state slots, captured graphs, sampler, command line — against
the plain CPU restatement."""
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import sodonex_fixtures as fx
from engine_helpers import agree, error, make_engine, portions, run, write_model
from oracle import sodonex as orc

pytestmark = pytest.mark.gpu
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
TOL = {torch.float32: 6e-5, torch.bfloat16: 3e-2}
DTYPES = [torch.float32, torch.bfloat16]


@pytest.mark.parametrize("dtype", DTYPES)
def test_residual_after_every_layer(dtype, monkeypatch):
    from llm_from_scratch_b200 import ops
    cfg = fx.config()
    w, ids, want, got = fx.weights(cfg, 1), fx.tokens(cfg, 90, 3), [], []
    orc.forward(cfg, w, ids, collect=want)
    plain = ops.shift_residual

    def spy(x, *a, **k):
        h = plain(x, *a, **k)
        if k.get("shift") is not None:                     # the residual moves on to the next layer
            got.append(k["x_out"][:90].double().cpu())
        return h

    eng = make_engine(cfg, w, dtype)
    monkeypatch.setattr(ops, "shift_residual", spy)
    run(eng, portions(ids, [90]))
    assert len(got) == len(want)
    for i, x in enumerate(want[:-1]):
        assert ((got[i + 1] - x).pow(2).mean(-1).sqrt().max() / x.std()).item() < TOL[dtype], i
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_whole_prompts_portions_and_single_tokens_give_the_same_logits(dtype):
    cfg = fx.config()
    w = fx.weights(cfg, 1)
    eng = make_engine(cfg, w, dtype)
    assert eng.model_runner.graphs          # single tokens replay captured graphs
    for n, sizes_list in ((150, [[150], [1], [2], [3, 1, 16], [64, 7, 2, 33], [37, 36, 38], [50, 100]]), (1, [[1]]),
                          (3, [[3], [2, 1], [1]]), (17, [[16, 1], [17]])):
        ids = fx.tokens(cfg, n, n)
        want = orc.forward(cfg, w, ids)
        for sizes in sizes_list:
            assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[dtype], sizes
    eng.exit()


def test_portions_gather_only_what_their_chunks_reach(monkeypatch):
    from llm_from_scratch_b200 import ops
    cfg = fx.config([fx.layer(None, chunk=20), fx.layer(None, chunk=0), fx.layer(None, chunk=90)])
    w, ids = fx.weights(cfg, 1), fx.tokens(cfg, 120, 3)
    want, totals = orc.forward(cfg, w, ids), []
    plain = ops.gather_rows
    monkeypatch.setattr(ops, "gather_rows", lambda *a, **k: (totals.append(a[4]), plain(*a, **k))[1])
    eng = make_engine(cfg, w, torch.float32)
    assert error(run(eng, portions(ids, [60, 10, 50]))["a"], want) < TOL[torch.float32]
    assert totals == [70, 70, 70, 70, 60, 60, 120, 120, 120, 120]       # keys and values; chunk 20 starts afresh at 60
    eng.exit()


VARIANTS = {
    "ones": fx.config([fx.layer(fx.moe(ff=8, experts=1, top=1), heads=1, kv_heads=1, dim=8, conv=1, rot_dims=2, chunk=1)], vocab=17, width=24),
    "odd": fx.config([fx.layer(fx.moe(ff=21, experts=6, top=6), heads=3, kv_heads=3, dim=7, conv=3, rot_dims=6, chunk=5),
                      fx.layer(fx.moe(ff=30, experts=3, top=2), heads=4, kv_heads=2, dim=11, conv=6, rot_dims=10, base=30.0, chunk=90)],
                     vocab=101, width=50, eps=1e-3, mult=1.0),
    "wide": fx.config([fx.layer(fx.moe(ff=64, experts=16, top=4), heads=4, kv_heads=2, dim=128, conv=4, rot_dims=64, chunk=70),
                       fx.layer(None, heads=18, kv_heads=9, dim=64, conv=2, rot_dims=16, chunk=64),
                       fx.layer(fx.moe(ff=256, experts=4, top=2), heads=16, kv_heads=1, dim=32, conv=3, rot_dims=32, chunk=33)],
                      vocab=260, width=256),
    "no chunks": fx.config([fx.layer(chunk=0), fx.layer(None, chunk=0, rot_dims=2)], embed_scale=0.5),
    "one long chunk": fx.config([fx.layer(chunk=1000, conv=17, kv_heads=6)], mult=2.0),
    "no rotation": fx.config([fx.layer(rot_dims=0, heads=2, kv_heads=1, dim=40), fx.layer(dim=56, rot_dims=56, conv=2)]),
    "no experts": fx.config([fx.layer(None), fx.layer(None, conv=1), fx.layer(None, chunk=7)]),
    "many taps": fx.config([fx.layer(conv=24, chunk=30)]),
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
        assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[dtype]
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_mixed_batches_on_pages_and_slots_that_are_used_again(dtype):
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
        assert error(got[name], orc.forward(cfg, w, ids[name])) < TOL[dtype], name
    assert eng.scheduler.block_manager.num_free_blocks == eng.model_runner.num_kv_blocks
    assert len(eng.scheduler.state_slots.free) == eng.model_runner.num_state_slots
    eng.exit()


KINDS = {"narrow": fx.config([fx.layer(chunk=48)], mult=1.0),
         "page": fx.config([fx.layer(heads=2, kv_heads=1, chunk=64, conv=2)], mult=1.0),
         "tensor cores": fx.config([fx.layer(None, heads=2, kv_heads=1, dim=128, rot_dims=32, chunk=100)], mult=1.0),
         "tensor cores, 64": fx.config([fx.layer(None, heads=4, kv_heads=2, dim=64, rot_dims=32, chunk=128, conv=3)], mult=1.0),
         "whole": fx.config([fx.layer(chunk=0)], mult=1.0),
         "two layers": fx.config([fx.layer(chunk=48), fx.layer(chunk=32)], mult=1.0)}


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("kind", sorted(KINDS))
def test_a_marked_key_counts_inside_its_chunk_only(kind, dtype):
    """One earlier token that stands out: at the first position of the query's chunk and just before it, beside page borders,
    inside the same portion and in an earlier one, the first of the sequence, far back; for queries inside a prompt and for decoded
    ones, at both ends of a chunk."""
    cfg = KINDS[kind]
    w = fx.marked_keys(cfg, fx.weights(cfg, 4))
    mixer = cfg["layers"][-1]["mixer"]
    n, chunk = 330, mixer["mask"]["size"] if mixer["mask"] else 0
    base = fx.plain_tokens(cfg, n, 8)
    eng = make_engine(cfg, w, dtype)
    seen = hidden = 0
    k = (n - 1) // chunk if chunk else 0
    ends = [k * chunk - 1, (k - 1) * chunk] if chunk else [255, 256]
    for last in sorted({n - 1, 40, *ends}):
        alone = orc.forward(cfg, w, base[:last] + [fx.SEEK])[last]
        start = last // chunk * chunk if chunk else 0
        for at in sorted({0, 15, 16, last - 17, start, start - 1, start - 30, last - 1} & set(range(last))):
            ids = list(base[:last]) + [fx.SEEK]
            ids[at] = fx.MARK
            want = orc.forward(cfg, w, ids)
            effect = ((want[last] - alone).pow(2).mean().sqrt() / want.std()).item()
            if at >= start:
                assert effect > 4 * TOL[torch.bfloat16], (last, at, effect)
                seen += 1
            elif len(cfg["layers"]) == 1 and at < start - mixer["conv"]:
                assert effect == 0.0
                hidden += 1
            for sizes in ([n], [last, 1], [last - 1, 2], [at + 1, 2, n]):
                got = run(eng, portions(ids, sizes))["a"]
                assert error(got[last:], want[last:]) < TOL[dtype], (last, at, sizes)
    assert seen >= 6 and (hidden >= 3 or chunk == 0 or len(cfg["layers"]) > 1)
    eng.exit()


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_first_tokens_after_a_slot_changed_hands(dtype):
    """A new request in the slot of an ended one: its first tokens have zeros before them, one by one and in portions."""
    cfg = fx.config()
    w = fx.weights(cfg, 6)
    a, b = fx.tokens(cfg, 30, 1), fx.tokens(cfg, 9, 2)
    want = orc.forward(cfg, w, b)
    eng = make_engine(cfg, w, dtype, max_requests=1)
    for sizes in ([1], [2], [9], [1, 3]):
        run(eng, portions(a, [30]))
        assert error(run(eng, portions(b, sizes))["a"], want) < TOL[dtype], sizes
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
    """Steps of new prompts replay a graph in bf16 (padded batches of unlike lengths, chunks, experts); steps with single
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
    from llm_from_scratch_b200.model.mixers import SoftmaxMoE
    cfg = fx.config([fx.layer(fx.moe(ff=64, experts=4, top=2), chunk=300)], width=128)
    w = fx.weights(cfg, 5)
    ids = fx.tokens(cfg, 700, 1)
    want = orc.forward(cfg, w, ids)
    for limit in (SoftmaxMoE.own_gemm_max_rows_per_expert, 1 << 20):
        eng = make_engine(cfg, w, torch.bfloat16, max_tokens=1024)
        eng.model_runner.model.layers[0].mlp.own_gemm_max_rows_per_expert = limit
        assert error(run(eng, portions(ids, [700]))["a"], want) < TOL[torch.bfloat16]
        eng.exit()


def test_a_prompt_of_thousands_of_tokens():
    """Several rows per CTA at the residual boundaries, segments of one sequence spread over many CTAs."""
    cfg = fx.config([fx.layer(fx.moe(16, 3, 1), chunk=500, heads=2, kv_heads=1), fx.layer(None, chunk=64, heads=2, kv_heads=2)], width=64)
    w = fx.weights(cfg, 5)
    ids = fx.tokens(cfg, 2600, 1)
    want = orc.forward(cfg, w, ids, torch.float32).double()
    eng = make_engine(cfg, w, torch.bfloat16, max_tokens=2688)
    for sizes in ([2600], [2301, 2, 297]):
        assert error(run(eng, portions(ids, sizes))["a"], want) < TOL[torch.bfloat16]
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
    la, lb = (orc.forward(cfg, w, ids) for ids in (a, b))
    pick = lambda x, y: {0: x[[0, 17]], 1: torch.stack([y[65], y[3], x[18]]), 3: torch.stack([x[19], y[69]])}
    want = pick(la, lb)
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
