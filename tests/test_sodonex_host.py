"""The Sodonex family without a GPU: configuration, registry, the key ranges of a step, and the plain restatement's mechanisms
against properties that do not depend on it."""
import itertools
import json

import numpy as np
import pytest
import torch

import sodonex_fixtures as fx
from llm_from_scratch_b200.engine import Sequence, metadata
from oracle import sodonex as orc


@pytest.fixture(autouse=True)
def _fresh():
    Sequence.block_size = 16
    Sequence.counter = itertools.count()
    Sequence.reference_exact = False


# ------------------------------------------------------------------------------ configuration, registry
def test_registry_and_round_trip():
    from llm_from_scratch_b200.model import SodonexConfig, SodonexLM, family_of, init_weights, resolve_config
    cfg = fx.config()
    parsed = resolve_config(cfg)
    assert isinstance(parsed, SodonexConfig) and family_of(cfg).model_cls is SodonexLM
    assert SodonexConfig.from_dict(json.loads(json.dumps(parsed.to_dict()))) == parsed
    assert parsed.layers[2].experts == 0 and parsed.layers[3].top == 1 and parsed.layers[1].chunk == 37 and parsed.residual_mult == 0.4
    assert resolve_config(fx.config([fx.layer(chunk=0)])).layers[0].chunk == 0
    w = init_weights(cfg, 0)
    assert w["l0.norm1"].shape == () and "l2.norm2" not in w and w["l1.mix.k.conv"].shape == (72, 2) and w["l3.mlp.e8.up"].shape == (24, 120)


@pytest.mark.parametrize("change", [
    dict(type="latent_attention"), dict(mlp={"kind": "dense", "ff": 8}), dict(mlp=fx.moe(experts=4, top=5)), dict(mlp=fx.moe(top=0)),
    dict(mixer=dict(fx.layer()["mixer"], vdim=8)), dict(mixer=dict(fx.layer()["mixer"], kv_heads=4)),
    dict(mixer=dict(fx.layer()["mixer"], rot=dict(dims=7, base=10.0))), dict(mixer=dict(fx.layer()["mixer"], rot=dict(dims=26, base=10.0))),
    dict(mixer=dict(fx.layer()["mixer"], conv=0))])
def test_configurations_that_cannot_be_served_are_refused(change):
    from llm_from_scratch_b200.model import SodonexConfig
    with pytest.raises(ValueError):
        SodonexConfig.from_dict(fx.config([dict(fx.layer(), **change)]))


def test_family_library_sources_exist():
    from llm_from_scratch_b200 import _build
    assert all((_build.CSRC / f"{n}.cu").exists() for n in _build.FAMILY_SOURCES["Sodonex"])


# ------------------------------------------------------------------------------------ key ranges of a step
def test_chunks_cut_the_contexts_of_portions():
    """A portion that starts at position p needs the keys from the start of p's chunk on."""
    lens = [(1, 9), (5, 5), (2, 30), (40, 100), (3, 103)]
    q, k = (np.concatenate([[0], np.cumsum(x)]).astype(np.int32) for x in zip(*lens))
    none = np.zeros(0, dtype=np.int64)
    p = metadata.StepMetadata(True, none, none, none, cu_seqlens_q=q, cu_seqlens_k=k).step_parts((8,), (1, 20, 25, 1000))
    assert p.num_single == 1 and sorted(p.ranges) == [8] and sorted(p.chunk_ranges) == [1, 20, 25, 1000]
    r = p.chunk_ranges
    assert np.diff(r[1].cu_k).tolist() == [5, 2, 40, 3] and not r[1].has_prefix
    assert np.diff(r[20].cu_k).tolist() == [5, 10, 40, 3] and r[20].has_prefix and r[20].max_seqlen_k == 40
    assert np.diff(r[25].cu_k).tolist() == [5, 5, 50, 3] and r[25].has_prefix and r[25].max_seqlen_k == 50
    assert r[1000].cu_k.tolist() == p.portion_cu_k.tolist()


def test_layers_find_their_range_by_chunk():
    from llm_from_scratch_b200.utils.context import KeyRange, Portions
    cu = torch.zeros(2, dtype=torch.int32)
    window, chunk = KeyRange(cu, 1, 1, False), KeyRange(cu, 2, 2, True)
    p = Portions(3, cu, cu, 3, 9, 9, True, cu, None, ranges={8: window}, chunk_ranges={8: chunk})
    assert p.keys(8) is window and p.keys(chunk=8) is chunk and p.keys().total_k == 9 and p.keys(chunk=5).has_prefix


# ---------------------------------------------------------------------------------- the restatement
def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_shift_mixes_the_token_before():
    x, s = _rand(4, 3), torch.tensor([0.0, 1.0, 0.25], dtype=torch.float64)
    y = orc.token_shift(x, s)
    assert torch.equal(y[:, 0], x[:, 0]) and torch.allclose(y[1:, 1], x[:-1, 1]) and y[0, 1] == 0
    assert torch.allclose(y[2, 2], 0.75 * x[2, 2] + 0.25 * x[1, 2])


def test_convolution_taps_end_at_the_token():
    u, w = _rand(5, 2), torch.tensor([[0.0, 0.0, 1.0], [1.0, 0.0, 0.0]], dtype=torch.float64)
    y = orc.short_conv(u, w)
    assert torch.equal(y[:, 0], u[:, 0]) and torch.equal(y[2:, 1], u[:3, 1]) and not y[:2, 1].any()


def test_rotation_pairs_halves_and_depends_on_distance_only():
    x = _rand(1, 1, 8).expand(40, 1, 8).contiguous()
    y = orc.rotate_half(x, 6, 100.0)
    assert torch.allclose(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    assert torch.allclose((y[3, 0] * y[10, 0]).sum(), (y[20, 0] * y[27, 0]).sum())
    e = torch.zeros(2, 1, 8, dtype=torch.float64)
    e[:, 0, 1] = 1
    turned = orc.rotate_half(e, 6, 100.0)[1, 0]
    assert turned.nonzero().flatten().tolist() == [1, 4] and torch.allclose(turned[4], torch.sin(torch.tensor(100.0).double() ** (-1 / 3)))


def test_chunks_count_from_position_zero():
    m = orc.chunk_mask(5, 9, 4, 3)
    assert [(~m[i]).nonzero().flatten().tolist() for i in range(5)] == [[3, 4], [3, 4, 5], [6], [6, 7], [6, 7, 8]]
    assert torch.equal(orc.chunk_mask(4, 4, 0, 0), torch.ones(4, 4, dtype=torch.bool).triu(1))


def test_weights_are_not_normalised():
    q, k, v = _rand(3, 2, 4), _rand(3, 1, 4, seed=1), _rand(3, 1, 4, seed=2)
    b = torch.tensor([0.5, -200.0]).double()
    o = orc.sigmoid_attention(q, k, v, 0.3, b)
    assert torch.allclose(o[1, 0], sum(torch.sigmoid(0.3 * (q[1, 0] @ k[j, 0]) + 0.5) * v[j, 0] for j in range(2)))
    assert o[:, 1].abs().max() < 1e-80


def test_norm_covers_the_whole_projection():
    x, w = _rand(4, 6), torch.arange(1.0, 7.0, dtype=torch.float64)
    y = orc.whole_norm(x, w, 1e-6)
    assert torch.allclose(y / w, x / (x.pow(2).mean(-1, keepdim=True) + 1e-6).sqrt())
    assert torch.allclose(orc.gain_norm(x, torch.tensor(2.0).double(), 1e-6), 2 * y / w)


def test_router_bias_counts_for_choice_and_weight():
    z = torch.tensor([1.0, 3.0, 2.0, -5.0]).double()
    (chosen, wts, margin), = orc.route(torch.ones(1, 1).double(), z[:, None], torch.tensor([0.0, 0.0, 0.0, 9.0]).double(), 2)
    assert chosen == [3, 1] and margin == pytest.approx(1.0)
    assert torch.allclose(wts, torch.softmax(torch.tensor([4.0, 3.0]).double(), 0))
    (chosen, wts, margin), = orc.route(torch.ones(1, 1).double(), z[:, None], torch.zeros(4).double(), 4)
    assert chosen == [1, 2, 0, 3] and margin == float("inf") and torch.allclose(wts.sum(), torch.tensor(1.0).double())


def test_a_layer_alone_does_not_cross_its_chunk_beyond_shift_and_convolution():
    cfg = fx.config([fx.layer(conv=3, chunk=20)])
    w = fx.weights(cfg, 3)
    a = fx.tokens(cfg, 30, 1)
    b = list(a)
    b[16] = (b[16] + 1) % cfg["vocab"]
    d = (orc.forward(cfg, w, a) - orc.forward(cfg, w, b)).abs().amax(-1)
    assert (d[16:20] > 0).all() and (d[20:] == 0).all()
    b = list(a)
    b[18] = (b[18] + 1) % cfg["vocab"]           # reaches the keys at 20 and 21: shifted at 19, two taps on
    d = (orc.forward(cfg, w, a) - orc.forward(cfg, w, b)).abs().amax(-1)
    assert (d[20:] > 0).all()


def test_fixture_margins_are_wide():
    cfg = fx.config()
    margins = []
    orc.forward(cfg, fx.weights(cfg, 1), fx.tokens(cfg, 60, 3), margins=margins)
    assert min(min(m) for m in margins) > 0.1
