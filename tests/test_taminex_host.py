"""The Taminex family without a GPU: configuration, registry, the two parts of a step, and the plain restatement's
mechanisms against properties that do not depend on it."""
import itertools
import json
import math

import numpy as np
import pytest
import torch

import taminex_fixtures as fx
from llm_from_scratch_b200.engine import SamplingParams, Sequence, metadata
from llm_from_scratch_b200.engine.scheduler import MixedScheduler
from oracle import taminex as orc


@pytest.fixture(autouse=True)
def _fresh():
    Sequence.block_size = 16
    Sequence.counter = itertools.count()
    Sequence.reference_exact = False


# ------------------------------------------------------------------------------ configuration, registry
def test_registry_and_round_trip():
    from llm_from_scratch_b200.model import TaminexConfig, TaminexLM, family_of, init_weights, resolve_config
    cfg = fx.config()
    parsed = resolve_config(cfg)
    assert isinstance(parsed, TaminexConfig) and family_of(cfg).model_cls is TaminexLM
    assert TaminexConfig.from_dict(json.loads(json.dumps(parsed.to_dict()))) == parsed
    assert [c.kind for c in parsed.layers] == ["latent_attention", "delta", "attention", "latent_attention", "delta"]
    assert parsed.layers[3].kv_from == 0 and parsed.layers[3].d_ff == 0 and parsed.layers[4].conv == 3
    w = init_weights(cfg, 0)
    assert "l0.mix.dkv" in w and "l3.mix.dkv" not in w and "l3.mlp.up" not in w and "head" not in w


@pytest.mark.parametrize("layers", [
    [dict(fx.delta(), type="other")], [dict(fx.delta(), mlp={"kind": "sparse", "ff": 8})], [fx.delta(heads=4, kv_heads=3)],
    [fx.attention(dims=7)], [fx.attention(dim=16, dims=32)], [fx.latent(kv_from=0)],
    [fx.delta(), fx.latent(kv_from=0)], [fx.latent(kv_rank=80), fx.latent(kv_rank=64, kv_from=0)],
    [fx.latent(), fx.latent(kv_from=0), fx.latent(kv_from=1)]])
def test_configurations_that_cannot_be_served_are_refused(layers):
    from llm_from_scratch_b200.model import TaminexConfig
    with pytest.raises(ValueError):
        TaminexConfig.from_dict(fx.config(layers))


def test_family_library_has_every_symbol_the_family_calls():
    from llm_from_scratch_b200 import _build
    assert all((_build.CSRC / f"{n}.cu").exists() for names in _build.FAMILY_SOURCES.values() for n in names)


# ------------------------------------------------------------------------------------ parts of a step
def _meta(lens):
    """lens: (tokens of the step, context length) per sequence."""
    q, k = (np.concatenate([[0], np.cumsum(x)]).astype(np.int32) for x in zip(*lens))
    none = np.zeros(0, dtype=np.int64)
    return metadata.StepMetadata(True, none, none, none, cu_seqlens_q=q, cu_seqlens_k=k)


def test_parts_of_a_step():
    p = _meta([(1, 9), (1, 1), (5, 5), (2, 30), (1, 4)]).step_parts()
    assert p.num_single == 2 and p.single_lens.tolist() == [9, 1] and p.portion_cu_k.tolist() == [0, 5, 35, 39]
    assert (p.max_seqlen_q, p.max_seqlen_k, p.has_prefix) == (5, 30, True)
    p = _meta([(7, 7), (3, 3)]).step_parts()
    assert p.num_single == 0 and not p.has_prefix and p.portion_cu_k.tolist() == [0, 7, 10]
    p = _meta([(1, 3), (1, 8)]).step_parts()
    assert p.num_single == 2 and p.max_seqlen_q == 0 and p.portion_cu_k.tolist() == [0]


def test_scheduler_puts_single_tokens_first():
    s = MixedScheduler(4, 64, 32, 16, eos=-1, num_state_slots=4)
    for n in (20, 1, 30):
        s.add_sequence(Sequence(list(range(n)), SamplingParams()))
    seqs, is_prefill = s.schedule()
    p = metadata.prepare_prefill(seqs, 16, tables_always=True).step_parts()
    assert is_prefill and [q.num_prompt_tokens for q in seqs] == [1, 20, 30]
    assert p.num_single == 1 and p.single_lens.tolist() == [1] and not p.has_prefix


# ---------------------------------------------------------------------------------- the restatement
def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_short_convolution_is_the_library_one():
    x, taps = _rand(11, 6), _rand(6, 4, seed=1)
    want = torch.nn.functional.conv1d(torch.nn.functional.pad(x.t()[None], (3, 0)), taps[:, None], groups=6)[0].t()
    assert torch.allclose(orc.short_conv(x, taps), want)


def test_delta_rule_overwrites_what_a_key_held():
    """Full strength, no decay: reading with the key just written returns the value just written, and another key's value
    stays as long as the keys are orthogonal."""
    k = torch.eye(4, dtype=torch.float64)[[0, 1, 0]].unsqueeze(1)
    v = _rand(3, 1, 5)
    ones, zero = torch.ones(3, 1, dtype=torch.float64), torch.zeros(3, 1, dtype=torch.float64)
    o, S = orc.delta_rule(k, k, v, ones, zero)
    assert torch.allclose(o[:, 0], v[:, 0]) and torch.allclose(S[0, 0], v[2, 0]) and torch.allclose(S[0, 1], v[1, 0])


def test_delta_rule_decays_before_it_reads_the_old_value():
    k = torch.eye(2, dtype=torch.float64)[[0, 0]].unsqueeze(1)
    v = torch.tensor([[[2.0]], [[0.0]]], dtype=torch.float64)
    beta, lg = torch.tensor([[1.0], [0.25]]).double(), torch.tensor([[0.0], [math.log(0.5)]], dtype=torch.float64)
    o, _ = orc.delta_rule(k, k, v, beta, lg)
    assert math.isclose(o[1, 0, 0].item(), 1.0 - 0.25 * 1.0)


def test_delta_rule_state_carries_over():
    q, k, v = orc.unit(_rand(9, 2, 4)), orc.unit(_rand(9, 2, 4, seed=1)), _rand(9, 4, 3, seed=2)
    beta, lg = torch.sigmoid(_rand(9, 4, seed=3)), -torch.rand(9, 4, dtype=torch.float64)
    whole, _ = orc.delta_rule(q, k, v, beta, lg)
    a, S = orc.delta_rule(q[:4], k[:4], v[:4], beta[:4], lg[:4])
    b, _ = orc.delta_rule(q[4:], k[4:], v[4:], beta[4:], lg[4:], S)
    assert torch.allclose(torch.cat([a, b]), whole)


def test_softplus_tails():
    x = torch.tensor([-800.0, -1.0, 0.0, 30.0, 800.0], dtype=torch.float64)
    assert torch.allclose(orc.softplus(x), torch.tensor([0.0, math.log1p(math.exp(-1)), math.log(2), 30.0, 800.0]).double())


def test_rotation_turns_neighbouring_channels_and_depends_on_distance_only():
    x = _rand(1, 1, 8).expand(40, 1, 8).contiguous()
    y = orc.rotate_pairs(x, 6, 100.0)
    assert torch.allclose(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    for i in range(3):
        assert torch.allclose(y[..., 2 * i:2 * i + 2].norm(dim=-1), x[..., 2 * i:2 * i + 2].norm(dim=-1))
    assert torch.allclose((y[3, 0] * y[10, 0]).sum(), (y[20, 0] * y[27, 0]).sum())
    a = 5 * 100.0 ** (-2 / 6)
    u, v = x[0, 0, 2].item(), x[0, 0, 3].item()
    assert math.isclose(y[5, 0, 2].item(), u * math.cos(a) - v * math.sin(a), rel_tol=1e-9)


def test_sink_takes_weight_and_gives_nothing():
    q, k, v = _rand(6, 2, 4), _rand(6, 1, 4, seed=1), torch.ones(6, 1, 3, dtype=torch.float64)
    sink = torch.tensor([0.3, -200.0], dtype=torch.float64)
    o = orc.causal_attention(q, k, v, 0.5, sink)
    assert torch.allclose(o[:, 1], torch.ones(6, 3, dtype=torch.float64))
    e = torch.exp(0.5 * (q[0, 0] @ k[0, 0]))
    assert torch.allclose(o[0, 0], (e / (e + math.exp(0.3))).expand(3))


def test_head_caps_and_scales():
    z = orc.head(torch.eye(2, dtype=torch.float64), torch.tensor([[2.0, 0.0], [0.0, 1e6]]).double(), 0.5, 10.0)
    assert math.isclose(z[0, 0].item(), 10 * math.tanh(0.1)) and math.isclose(z[1, 1].item(), 10.0)


def test_shared_latent_rows_are_the_source_layers():
    """The sharing layer has no down-projection and still attends."""
    cfg = fx.config([fx.latent(), fx.latent(kv_from=0)])
    w = fx.weights(cfg, 0)
    assert "l1.mix.dkv" not in w
    full, one = [], []
    orc.forward(cfg, w, [1, 2, 3, 4], collect=full)
    orc.forward(dict(cfg, layers=cfg["layers"][:1]), w, [1, 2, 3, 4], collect=one)
    assert torch.equal(full[0], one[0]) and not torch.allclose(full[1], full[0])
