"""The host side of mixed batches and the Nabalix family without a GPU: configuration, registry, scheduler, state
slots, step metadata, and the plain restatement against itself."""
import itertools
import json
import random

import numpy as np
import pytest
import torch

import nabalix_fixtures as fx
from llm_from_scratch_b200.engine import NativeBlockManager, SamplingParams, Sequence, metadata
from llm_from_scratch_b200.engine.llm_engine import LLMEngine
from llm_from_scratch_b200.engine.scheduler import MixedScheduler, StateSlots
from oracle import nabalix as orc


@pytest.fixture(autouse=True)
def _fresh():
    Sequence.block_size = 16
    Sequence.counter = itertools.count()
    Sequence.reference_exact = False


# ------------------------------------------------------------------------------ configuration, registry
def test_registry_chooses_the_family_by_architecture():
    from llm_from_scratch_b200.model import (EngineTransformerLM, ModelConfig, NabalixConfig, NabalixLM, family_of,
                                             init_weights, resolve_config)
    cfg = fx.config()
    assert isinstance(resolve_config(cfg), NabalixConfig) and family_of(cfg).model_cls is NabalixLM
    plain = dict(vocab_size=64, d_model=32, num_heads=4, num_layers=1, d_ff=16)
    assert isinstance(resolve_config(plain), ModelConfig) and family_of(plain).model_cls is EngineTransformerLM
    with pytest.raises(ValueError, match="unknown architecture"):
        family_of({"architecture": "Nothing"})
    assert set(init_weights(plain, 0)) > {"token_embeddings.weight", "lm_head.weight"}


def test_configuration_round_trip_and_rejections():
    from llm_from_scratch_b200.model import NabalixConfig
    cfg = fx.config()
    parsed = NabalixConfig.from_dict(cfg)
    assert NabalixConfig.from_dict(json.loads(json.dumps(parsed.to_dict()))) == parsed
    assert parsed.layers[1].d_ff == 0 and parsed.layers[2].window == 130 and parsed.num_layers == 3
    for change in (dict(type="other"), dict(mlp={"kind": "sparse", "ff": 8, "limit": 1.0})):
        bad = fx.config([dict(fx.layer(), **change)])
        with pytest.raises(ValueError):
            NabalixConfig.from_dict(bad)
    with pytest.raises(ValueError):
        NabalixConfig.from_dict(fx.config([fx.layer(heads=4, kv_heads=3)]))


def test_model_folder_loads(tmp_path):
    from safetensors.torch import save_file
    from llm_from_scratch_b200.utils.loader import load_model_dir
    cfg = fx.config()
    w = fx.weights(cfg)
    (tmp_path / "config.json").write_text(json.dumps(cfg))
    save_file(w, str(tmp_path / "model.safetensors"))
    got, state = load_model_dir(str(tmp_path))
    assert got == cfg and state.keys() == w.keys() and all(torch.equal(state[k], w[k]) for k in w)


# ------------------------------------------------------------------------------------------ scheduler
def test_state_slots_are_handed_out_once_and_come_back():
    slots = StateSlots(2)
    a, b, c = Sequence([1]), Sequence([1]), Sequence([1])
    slots.take(a)
    slots.take(a)
    slots.take(b)
    assert sorted((a.state_slot, b.state_slot)) == [0, 1]
    with pytest.raises(IndexError):
        slots.take(c)
    freed = a.state_slot
    slots.give_back(a)
    slots.give_back(a)
    slots.take(c)
    assert c.state_slot == freed and a.state_slot == -1 and not slots.free


def test_pool_without_prefix_caching_never_shares_blocks():
    bm = NativeBlockManager(8, 16, prefix_caching=False)
    a, b = Sequence(list(range(33))), Sequence(list(range(33)))
    bm.allocate(a)
    bm.allocate(b)
    assert len(set(a.block_table + b.block_table)) == 6 and b.num_cached_tokens == 0
    bm.grow(a, 48)
    assert len(a.block_table) == 3
    bm.grow(a, 50)
    assert len(a.block_table) == 4 and bm.num_free_blocks == 1
    bm.deallocate(a)
    assert bm.num_free_blocks == 5


class FakeRunner:
    """Executes scheduled batches on the host: the next token is a hash of the whole prefix, and it checks that
    exactly the uncached tokens arrive, that tables cover them and that slots are held by one sequence each."""

    mixed_batches = True

    def __init__(self, blocks, slots, block_size=16, budget=64):
        self.num_kv_blocks, self.num_state_slots, self.bs, self.budget = blocks, slots, block_size, budget
        self.state, self.batches, self.max_model_length = {}, [], 4096

    @staticmethod
    def token(ids):
        return hash(tuple(ids)) % 97

    def run(self, seqs, is_prefill):
        out, total = [], 0
        slots = [s.state_slot for s in seqs]
        assert len(set(slots)) == len(slots) and min(slots) >= 0
        blocks = [b for s in seqs for b in s.block_table]
        assert len(set(blocks)) == len(blocks)
        if is_prefill:
            m = metadata.prepare_prefill(seqs, self.bs, tables_always=True)
            assert m.block_tables is not None and m.state_slots.tolist() == slots
            lens = np.diff(m.cu_seqlens_q)
            assert m.input_ids.tolist() == [t for s in seqs for t in s.token_ids[s.num_cached_tokens:s.step_end]]
            assert np.diff(m.cu_seqlens_k).tolist() == [s.step_end for s in seqs]
            singles = [n == 1 for n in lens]
            assert singles == sorted(singles, reverse=True)          # single tokens lead the batch
        else:
            m = metadata.prepare_decode(seqs, self.bs)
            lens = [1] * len(seqs)
            assert m.context_lens.tolist() == [s.num_tokens for s in seqs] == [s.num_cached_tokens + 1 for s in seqs]
        for s, n in zip(seqs, lens):
            assert n == s.step_end - s.num_cached_tokens > 0
            # the state a slot carries is that of exactly the cached tokens
            assert s.num_cached_tokens == 0 or self.state[s.state_slot] == tuple(s.token_ids[:s.num_cached_tokens])
            self.state[s.state_slot] = tuple(s.token_ids[:s.step_end])
            total += int(n)
            out.append(self.token(s.token_ids[:s.step_end]))
        assert total <= self.budget
        self.batches.append((len(seqs), is_prefill, total))
        return out

    def exit(self):
        pass


@pytest.mark.parametrize("blocks,budget,slots", [(200, 64, 4), (200, 7, 4), (12, 64, 4), (9, 20, 3)])
def test_mixed_scheduler_serves_every_request_exactly(blocks, budget, slots):
    rng = random.Random(blocks * budget)
    runner = FakeRunner(blocks, slots, budget=budget)
    eng = LLMEngine(dict(block_size=16, max_num_sequences=slots, max_num_batched_tokens=budget, eos=-1), runner=runner)
    assert isinstance(eng.scheduler, MixedScheduler)
    prompts = [[rng.randrange(97) for _ in range(rng.choice([1, 2, 15, 16, 17, 40, 70]))] for _ in range(12)]
    out = eng.generate(prompts, [SamplingParams(temperature=0.0, max_tokens=rng.choice([2, 9, 30]), ignore_eos=True)
                                 for _ in prompts])["token_ids"]
    for p, got in zip(prompts, out):
        ids = list(p)
        for t in got:
            assert t == runner.token(ids)
            ids.append(t)
    bm = eng.scheduler.block_manager
    assert bm.num_free_blocks == blocks and len(eng.scheduler.state_slots.free) == slots
    if budget < 40:        # prompts were read in portions beside decoded tokens
        assert any(p and n > 1 for n, p, _ in runner.batches)


def test_a_request_that_can_never_fit_is_reported():
    eng = LLMEngine(dict(block_size=16, max_num_sequences=2, max_num_batched_tokens=64, eos=-1), runner=FakeRunner(2, 2))
    with pytest.raises(RuntimeError, match="nothing schedulable"):
        eng.generate([list(range(40))], SamplingParams(temperature=0.0, max_tokens=4))


def test_feeding_tokens_and_dropping_requests():
    s = MixedScheduler(4, 64, 6, 16, -1, num_state_slots=2)
    a, b = Sequence([]), Sequence([])
    batch, is_prefill = s.feed([(a, [1, 2, 3]), (b, [9])])
    assert batch == [b, a] and is_prefill
    assert [(x.num_cached_tokens, x.step_end) for x in (a, b)] == [(0, 3), (0, 1)]
    s.fed(batch)
    batch, is_prefill = s.feed([(a, [4]), (b, [8])])
    assert not is_prefill and a.last_token == 4 and a.num_tokens == 4
    s.fed(batch)
    with pytest.raises(IndexError):
        s.feed([(Sequence([]), [1])])
    s.drop(a)
    c = Sequence([])
    s.feed([(c, [5] * 20)])
    assert c.state_slot >= 0
    assert len(c.block_table) == 2


# ------------------------------------------------------------------------- the restatement against itself
def test_restatement_recurrence_resumes_from_its_state_and_matches_the_closed_form():
    g = torch.Generator().manual_seed(0)
    q, f, v = torch.randn(9, 2, 4, generator=g).double(), torch.rand(9, 2, 4, generator=g).double(), torch.randn(
        9, 2, 3, generator=g).double()
    o, S = orc.gated_recurrence(q, f, v)
    o1, S1 = orc.gated_recurrence(q[:5], f[:5], v[:5])
    o2, S2 = orc.gated_recurrence(q[5:], f[5:], v[5:], S1)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(S2, S)
    t = 6                                          # S_t = sum_j prod_{j < s <= t} f_s (1 - f_j) v_j^T
    want = sum(torch.prod(f[j + 1:t + 1], 0)[:, :, None] * (1 - f[j])[:, :, None] * v[j][:, None, :] for j in range(t + 1))
    assert torch.allclose(torch.einsum("hkv,hk->hv", want, q[t]), o[t])


def test_restatement_attention_by_scalars():
    """One query of the matrix form against loops over heads and keys."""
    g = torch.Generator().manual_seed(1)
    H, G, dk, dv, n, window, cap, scale = 4, 2, 3, 5, 8, 3, 2.0, 0.7
    q, k, v = (torch.randn(*s, generator=g).double() for s in ((n, H, dk), (n, G, dk), (n, G, dv)))
    r1, r2, T = torch.rand(H, generator=g).double(), torch.rand(H, generator=g).double(), torch.randn(H, H, generator=g).double()
    got = orc.attention(q, k, v, scale, cap, r1, r2, T, window)
    i = 6
    s = {(h, j): cap * np.tanh(float(q[i, h] @ k[j, h // 2]) * scale / cap) - float(r1[h]) * np.log(1 + float(r2[h]) * (i - j))
         for h in range(H) for j in range(n)}
    for h in range(H):
        m = {j: sum(float(T[h, x]) * s[x, j] for x in range(H)) for j in (4, 5, 6)}
        z = sum(np.exp(x) for x in m.values())
        want = sum(np.exp(m[j]) / z * v[j, h // 2] for j in m)
        assert torch.allclose(want, got[i, h])


def test_restatement_streams_by_scalars():
    g = torch.Generator().manual_seed(2)
    X, y, mix, w = torch.randn(2, 1, 3, generator=g), torch.randn(1, 3, generator=g), torch.randn(2, 2, generator=g), torch.randn(
        2, generator=g)
    got = orc.streams_write(X, y, mix, w)
    assert torch.allclose(got[1], mix[0, 1] * X[0] + mix[1, 1] * X[1] + w[1] * y)
