"""The Meresun family without a GPU: configuration, registry, the key ranges of a step, and the plain restatement's mechanisms
against properties that do not depend on it."""
import itertools
import json
import math

import numpy as np
import pytest
import torch

import meresun_fixtures as fx
from llm_from_scratch_b200.engine import Sequence, metadata
from oracle import meresun as orc


@pytest.fixture(autouse=True)
def _fresh():
    Sequence.block_size = 16
    Sequence.counter = itertools.count()
    Sequence.reference_exact = False


# ------------------------------------------------------------------------------ configuration, registry
def test_registry_and_round_trip():
    from llm_from_scratch_b200.model import MeresunConfig, MeresunLM, family_of, init_weights, resolve_config
    cfg = fx.config()
    parsed = resolve_config(cfg)
    assert isinstance(parsed, MeresunConfig) and family_of(cfg).model_cls is MeresunLM
    assert MeresunConfig.from_dict(json.loads(json.dumps(parsed.to_dict()))) == parsed
    assert parsed.layers[2].scaling is None and parsed.layers[2].d_ff == 0 and parsed.layers[1].experts == 12
    assert parsed.layers[0].scaling.magnitude == pytest.approx(0.1 * math.log(4.0) + 1)
    w = init_weights(cfg, 0)
    assert "l0.mlp.act" in w and "l1.mlp.e11.down" in w and "l2.rg2" not in w and w["side.embed"].shape == (131, 80)


def test_order_of_layer_runs():
    from llm_from_scratch_b200.model import resolve_config
    for loop in ((1, 3, 2), (0, 4, 3), (3, 4, 4), (0, 1, 1), None):
        cfg = fx.config(loop=loop)
        assert resolve_config(cfg).layer_runs() == orc.layer_runs(cfg)
    assert orc.layer_runs(fx.config(loop=(1, 3, 2))) == [(0, False), (1, False), (2, False), (1, True), (2, False), (3, False)]


@pytest.mark.parametrize("change", [
    dict(layers=[dict(fx.layer(), type="other")]), dict(layers=[fx.layer({"kind": "sparse", "ff": 8})]),
    dict(layers=[fx.layer(fx.moe(groups=(5, 2)))]), dict(layers=[fx.layer(fx.moe(experts=8, top=5, groups=(2, 1)))]),
    dict(layers=[fx.layer(rot_dim=7)]), dict(loop=(2, 1, 2)), dict(loop=(0, 9, 2)), dict(groups=7)])
def test_configurations_that_cannot_be_served_are_refused(change):
    from llm_from_scratch_b200.model import MeresunConfig
    with pytest.raises(ValueError):
        MeresunConfig.from_dict(fx.config(**change))


def test_family_library_sources_exist():
    from llm_from_scratch_b200 import _build
    assert all((_build.CSRC / f"{n}.cu").exists() for n in _build.FAMILY_SOURCES["Meresun"])


# ------------------------------------------------------------------------------------ key ranges of a step
def test_windows_cut_the_contexts_of_portions():
    """A portion of q tokens at the end of k needs its last min(k, q + window - 1) keys."""
    lens = [(1, 9), (5, 5), (2, 30), (40, 100)]
    q, k = (np.concatenate([[0], np.cumsum(x)]).astype(np.int32) for x in zip(*lens))
    none = np.zeros(0, dtype=np.int64)
    p = metadata.StepMetadata(True, none, none, none, cu_seqlens_q=q, cu_seqlens_k=k).step_parts((1, 8, 1000))
    assert p.num_single == 1 and sorted(p.ranges) == [1, 8, 1000]
    assert p.ranges[1].cu_k.tolist() == [0, 5, 7, 47] and not p.ranges[1].has_prefix and p.ranges[1].max_seqlen_k == 40
    assert p.ranges[8].cu_k.tolist() == [0, 5, 14, 61] and p.ranges[8].has_prefix and p.ranges[8].max_seqlen_k == 47
    assert p.ranges[1000].cu_k.tolist() == p.portion_cu_k.tolist() == [0, 5, 35, 135]


# ------------------------------------------------------------------------------------------ frequencies
@pytest.mark.parametrize("dims,base,scaling", [(8, 1000.0, fx.YARN), (64, 5e5, dict(factor=8.0, original=4096, fast=32.0, slow=1.0)),
                                               (16, 1e4, dict(factor=40.0, original=7, fast=1.0, slow=1.0)), (2, 50.0, fx.YARN),
                                               (32, 1e4, None)])
def test_stretched_frequencies(dims, base, scaling):
    from llm_from_scratch_b200 import ops
    want, size = orc.rotary_frequencies(dims, base, scaling)
    y = ops.YarnScaling(**{k: float(v) for k, v in scaling.items()}) if scaling else None
    r = ops.Rotation(base, dims, "cpu", y)
    assert torch.allclose(r.freq, want, rtol=1e-12) and r.magnitude == pytest.approx(size)
    if scaling:
        plain = orc.rotary_frequencies(dims, base)[0]
        ratio = want / plain
        assert (ratio <= 1 + 1e-12).all() and (ratio >= 1 / scaling["factor"] - 1e-12).all()


def test_ramp_leaves_fast_pairs_and_stretches_slow_ones():
    s = dict(factor=16.0, original=4096, fast=32.0, slow=1.0)
    f, size = orc.rotary_frequencies(64, 10000.0, s)
    plain, one = orc.rotary_frequencies(64, 10000.0)
    turns = 4096 * plain / (2 * math.pi)
    assert torch.allclose(f[turns > 40], plain[turns > 40]) and torch.allclose(f[turns < 0.8], plain[turns < 0.8] / 16)
    assert one == 1.0 and size == pytest.approx(1.2772588722)


# ---------------------------------------------------------------------------------- the restatement
def _rand(*shape, seed=0):
    return torch.randn(*shape, generator=torch.Generator().manual_seed(seed), dtype=torch.float64)


def test_window_counts_the_token_itself():
    m = orc.window_mask(3, 10, 4, 7)
    assert [(~m[i]).nonzero().flatten().tolist() for i in range(3)] == [[4, 5, 6, 7], [5, 6, 7, 8], [6, 7, 8, 9]]
    assert (~orc.window_mask(2, 2, 1, 0)).nonzero().tolist() == [[0, 0], [1, 1]]


def test_sink_takes_weight_and_gives_nothing():
    q, k, v = _rand(6, 2, 4), _rand(6, 2, 4, seed=1), torch.ones(6, 2, 3, dtype=torch.float64)
    o = orc.windowed_attention(q, k, v, 0.5, torch.tensor([0.3, -200.0]).double(), 3)
    assert torch.allclose(o[:, 1], torch.ones(6, 3, dtype=torch.float64))
    e = torch.exp(0.5 * (q[0, 0] @ k[0, 0]))
    assert torch.allclose(o[0, 0], (e / (e + math.exp(0.3))).expand(3))


def test_rotation_depends_on_distance_only_and_scales_scores():
    x = _rand(1, 1, 8).expand(40, 1, 8).contiguous()
    y = orc.rotate_pairs(x, 6, 100.0)
    assert torch.allclose(y[0], x[0]) and torch.equal(y[..., 6:], x[..., 6:])
    z = orc.rotate_pairs(x, 6, 100.0, fx.YARN)
    assert torch.allclose((z[3, 0] * z[10, 0]).sum(), (z[20, 0] * z[27, 0]).sum())
    assert torch.allclose(z[0, 0, :6], x[0, 0, :6] * (0.1 * math.log(4.0) + 1))


def test_group_norm_parts_are_independent():
    x, w = _rand(4, 12), torch.ones(12, dtype=torch.float64)
    y = orc.group_norm(x, w, 3, 1e-6)
    assert torch.allclose(y[:, 4:8], orc.rms(x[:, 4:8], 1e-6)) and torch.allclose(orc.group_norm(x, w, 1, 1e-6), orc.rms(x, 1e-6))


def test_poly_norm_terms():
    z, c = _rand(3, 50), torch.tensor([2.0, 0.0, 0.0, 0.5]).double()
    assert torch.allclose(orc.poly_norm(z, c, 1e-6), 2 * orc.rms(z, 1e-6) + 0.5)
    y = orc.poly_norm(z, torch.tensor([0.0, 1.0, -1.0, 0.0]).double(), 0.0)
    assert torch.allclose(y, z ** 2 / (z ** 4).mean(-1, keepdim=True).sqrt() - z ** 3 / (z ** 6).mean(-1, keepdim=True).sqrt())


def test_router_groups_and_correction():
    """Choice by corrected scores inside the best groups, weights from the plain ones; left-out groups never win, also
    when every choice score is negative."""
    h = torch.eye(1, dtype=torch.float64)
    z = torch.tensor([2.0, -1.0, 1.0, 1.5, -3.0, 3.0], dtype=torch.float64)
    (chosen, wts, _), = orc.route(h, z[:, None], torch.zeros(6).double(), 3, 1, 2)
    assert chosen == [2, 3]                               # group scores: 0.88 + 0.27, 0.73 + 0.82, 0.05 + 0.95
    s = torch.sigmoid(z[[2, 3]])
    assert torch.allclose(wts, s / s.sum())
    (chosen, wts, _), = orc.route(h, z[:, None], torch.tensor([-9.0, -9, -2, -2, -3, -3]).double(), 3, 1, 2)
    assert chosen == [2, 3] and torch.allclose(wts, s / s.sum())
    (chosen, _, margin), = orc.route(h, z[:, None], torch.tensor([0.0, 0, 0, 0, 0.9, 0]).double(), 3, 2, 1)
    assert chosen == [5] and margin == pytest.approx(float(torch.sigmoid(z[5]) - torch.sigmoid(z[4])) - 0.9, abs=1e-6)


def test_gelu_and_clamped_glu():
    z = torch.linspace(-6, 6, 41, dtype=torch.float64)
    assert torch.allclose(orc.gelu_tanh(z), torch.nn.functional.gelu(z, approximate="tanh"))
    g, u = torch.tensor([5.0, -1.0]).double(), torch.tensor([-7.0, 0.5]).double()
    want = [1.5 * (1 / (1 + math.exp(-1.702 * 1.5))) * (-1.5 + 1), -1.0 * (1 / (1 + math.exp(1.702))) * 1.5]
    assert torch.allclose(orc.clamped_glu(g, u, 1.5), torch.tensor(want).double())


def test_a_loop_adds_the_embedding_before_its_later_passes():
    cfg = fx.config([fx.layer(fx.dense())], loop=(0, 1, 2))
    w = fx.weights(cfg, 0)
    once, twice = [], []
    orc.forward(dict(cfg, loop=None), w, [1, 2, 3], collect=once)
    orc.forward(cfg, w, [1, 2, 3], collect=twice)
    assert torch.equal(once[0], twice[0]) and len(twice) == 2
