"""Kernels behind the Taminex family, each alone, against the plain CPU restatement."""
import math

import pytest
import torch

from oracle import attention as att
from oracle import taminex as orc

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 2e-2}


def gen(seed=0):
    return torch.Generator().manual_seed(seed)


def close(got, want, tol):
    """Largest difference in units of the element's magnitude plus the reference's rms."""
    want = want.double()
    err = ((got.double().cpu() - want).abs() / (want.abs() + want.pow(2).mean().sqrt() + 1e-30)).max().item()
    assert err <= tol, err


def cu(lens):
    return torch.tensor([0] + torch.tensor(lens).cumsum(0).tolist(), dtype=torch.int32)


def tables(lens, bs, seed=0, spare=3):
    """(block tables, number of blocks) with shuffled blocks for contexts of these lengths."""
    need = [(n + bs - 1) // bs for n in lens]
    ids = torch.randperm(sum(need) + spare, generator=gen(seed)).int()
    bt = torch.full((len(lens), max(need + [1])), -1, dtype=torch.int32)
    at = 0
    for i, n in enumerate(need):
        bt[i, :n] = ids[at:at + n]
        at += n
    return bt, sum(need) + spare


def rows_of(pool, bt, i, n):
    """The n cached rows of sequence i."""
    bs = pool.shape[1]
    flat = pool.reshape(-1, *pool.shape[2:])
    return flat[[int(bt[i, j // bs]) * bs + j % bs for j in range(n)]]


# ------------------------------------------------------------------------------------------- residual
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [64, 100, 333, 1024, 4096, 6144, 10000])
def test_residual_norm(d, dtype):
    from llm_from_scratch_b200 import ops
    T, eps = 7, 1e-4
    g = gen(d)
    embed = torch.randn(50, d, generator=g).to(dtype)
    toks = torch.randint(0, 50, (T,), generator=g)
    y = (3 * torch.randn(T, d, generator=g)).to(dtype)
    w, fw = torch.rand(d, generator=g), torch.rand(d, generator=g)
    x = torch.full((T, d), 7.0, device="cuda")
    h = ops.residual_norm(x, eps, dtype, tokens=toks.cuda(), embed=embed.cuda())
    assert torch.equal(x.cpu(), embed[toks].float()) and torch.equal(h.cpu(), embed[toks])
    want = embed[toks].double() + orc.rms_norm(y.double(), w.double(), eps)
    h = ops.residual_norm(x, eps, dtype, y=y.cuda(), norm_w=w.cuda())
    close(x, want, 1e-5)
    assert torch.equal(h.cpu(), x.cpu().to(dtype))
    h = ops.residual_norm(x, eps, dtype, y=y.cuda(), norm_w=w.cuda(), final_w=fw.cuda())
    want = want + orc.rms_norm(y.double(), w.double(), eps)
    close(x, want, 1e-5)
    close(h, orc.rms_norm(want, fw.double(), eps), TOL[dtype])
    ops.check_status()


# --------------------------------------------------------------------------------------- head norm, rotation
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,G,D,Dv,dims", [(4, 2, 64, 64, 32), (6, 3, 48, 20, 48), (3, 1, 130, 7, 2), (8, 8, 128, 128, 64),
                                            (2, 1, 256, 64, 0), (5, 5, 17, 9, 16)])
def test_head_norm_rope_store(Hq, G, D, Dv, dims, dtype):
    from llm_from_scratch_b200 import ops
    g, T, bs, base = gen(D), 11, 16, 5000.0
    widths = [Hq * D, G * D, G * Dv]
    starts = [0, (widths[0] + 7) // 8 * 8]
    starts.append(starts[1] + (widths[1] + 7) // 8 * 8)
    proj = torch.randn(T, starts[2] + (widths[2] + 7) // 8 * 8, generator=g).to(dtype)
    q, k, v = (proj[:, s:s + w] for s, w in zip(starts, widths))
    wq, wk = torch.rand(D, generator=g) + 0.5, torch.rand(D, generator=g) + 0.5
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4095, 70001, 1 << 20, 5, 6])
    slots = torch.tensor([3, -1, 17, 16, 40, 5, 6, 7, 8, 9, 31])
    kc, vc = torch.zeros(3, bs, G, D, dtype=dtype, device="cuda"), torch.zeros(3, bs, G, Dv, dtype=dtype, device="cuda")
    pc = proj.cuda()
    qo, ko = ops.head_norm_rope_store(*(pc[:, s:s + w] for s, w in zip(starts, widths)), wq.cuda(), wk.cuda(), 1e-5,
                                      ops.rotary_frequencies(base, dims, "cuda"), pos.cuda(), kc, vc, slots.cuda())
    ops.check_status()
    for got, x, w, H in ((qo, q, wq, Hq), (ko, k, wk, G)):
        n = orc.rms_norm(x.double().reshape(T, H, D), w.double(), 1e-5)
        want = torch.cat([orc.rotate_pairs(n[t:t + 1], dims, base, int(pos[t])) for t in range(T)])
        close(got, want, TOL[dtype])
    for t in range(T):
        if slots[t] >= 0:
            assert torch.equal(kc.view(-1, G, D)[slots[t]], ko[t])
            assert torch.equal(vc.view(-1, G, Dv)[slots[t]].cpu().reshape(-1), v[t])
    used = set(slots[slots >= 0].tolist())
    rest = [i for i in range(3 * bs) if i not in used]
    assert not kc.view(-1, G, D)[rest].any() and not vc.view(-1, G, Dv)[rest].any()


# ------------------------------------------------------------------------------------------ attention sinks
def sink_for(H, seed):
    s = 2 * torch.randn(H, generator=gen(seed))
    s[0], s[-1] = 7.0, -60.0                     # one that takes nearly everything, one that takes nothing
    return s


SINK_SHAPES = [(4, 2, 128, 128), (8, 2, 64, 64), (6, 3, 64, 64), (3, 1, 32, 32), (5, 5, 128, 128), (6, 2, 48, 40), (2, 1, 64, 256)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("paged", [False, True])
@pytest.mark.parametrize("Hq,G,D,Dv", SINK_SHAPES)
def test_prefill_with_a_sink(Hq, G, D, Dv, paged, dtype):
    from llm_from_scratch_b200 import ops
    g, bs, scale = gen(D), 64 if D == 64 else 16, 1.3 * D ** -0.5
    qlens = [1, 70, 2, 300]
    klens = [n + (e if paged else 0) for n, e in zip(qlens, (5, 0, 200, 64))]
    T = sum(qlens)
    q = torch.randn(T, Hq, D, generator=g).to(dtype)
    ks = [torch.randn(n, G, D, generator=g).to(dtype) for n in klens]
    vs = [torch.randn(n, G, Dv, generator=g).to(dtype) for n in klens]
    sink = sink_for(Hq, 1)
    kw = {}
    if paged:
        bt, nb = tables(klens, bs)
        kc, vc = torch.zeros(nb, bs, G, D, dtype=dtype), torch.zeros(nb, bs, G, Dv, dtype=dtype)
        for i, n in enumerate(klens):
            for j in range(n):
                b, o = int(bt[i, j // bs]), j % bs
                kc[b, o], vc[b, o] = ks[i][j], vs[i][j]
        args = (None, None)
        kw = dict(k_cache=kc.cuda(), v_cache=vc.cuda(), block_tables=bt.cuda())
    else:
        args = (torch.cat(ks).cuda(), torch.cat(vs).cuda())
    cq, ck = cu(qlens).cuda(), cu(klens).cuda()
    want = torch.cat([orc.causal_attention(q[a:b].double(), ks[i].double(), vs[i].double(), scale, sink.double(),
                                           klens[i] - qlens[i])
                      for i, (a, b) in enumerate(zip(cu(qlens)[:-1].tolist(), cu(qlens)[1:].tolist()))])
    for rows in (0, ops.prefill_tile_rows(Hq, G, D, Dv, dtype, paged=paged)):
        plan = ops.prefill_plan(cq, T, max(qlens), rows)
        got = ops.prefill_varlen(q.cuda(), *args, cq, ck, max(qlens), max(klens), scale, plan=plan, sink=sink.cuda(), **kw)
        ops.check_status()
        assert (got.double().cpu() - want).abs().max() <= TOL[dtype]
        assert want[:, 0].abs().max() < 1.0 and want[:, -1].abs().max() > 0.5


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("Hq,G,D,Dv", SINK_SHAPES)
@pytest.mark.parametrize("batch", [5, 40])
def test_decode_with_a_sink(Hq, G, D, Dv, bs, batch, dtype):
    """One launch that merges split contexts inside (small batches) and the separate merge; contexts of one token, at
    block borders, and long enough to be cut over many CTAs; an empty row."""
    from llm_from_scratch_b200 import ops
    g, scale = gen(D + bs), D ** -0.5
    lens = ([1, 16, 17, 0, 2100, 64, 65, 5] * 8)[:batch]
    bt, nb = tables(lens, bs)
    kc = torch.randn(nb, bs, G, D, generator=g).to(dtype)
    vc = torch.randn(nb, bs, G, Dv, generator=g).to(dtype)
    q, sink = torch.randn(batch, Hq, D, generator=g).to(dtype), sink_for(Hq, 2)
    got = ops.paged_decode_gqa(q.cuda(), kc.cuda(), vc.cuda(), bt.cuda(), torch.tensor(lens).cuda(), scale, sink=sink.cuda())
    ops.check_status()
    for i, n in enumerate(lens):
        if n == 0:
            assert not got[i].any()
            continue
        want = orc.causal_attention(q[i:i + 1].double(), rows_of(kc, bt, i, n).double(), rows_of(vc, bt, i, n).double(), scale,
                                    sink.double(), n - 1)
        assert (got[i].double().cpu() - want[0]).abs().max() <= TOL[dtype], (i, n)


def test_block_sizes_agree_without_a_sink():
    """The decode kernel walks 16-token blocks inside larger pages."""
    from llm_from_scratch_b200 import ops
    g, lens = gen(3), [300, 64, 1, 777]
    bt64, nb = tables(lens, 64)
    kc, vc = (torch.randn(nb, 64, 2, 128, generator=g).bfloat16().cuda() for _ in range(2))
    q, n = torch.randn(4, 8, 128, generator=g).bfloat16().cuda(), torch.tensor(lens).cuda()
    bt16 = torch.where(bt64[:, :, None] < 0, -1, bt64[:, :, None] * 4 + torch.arange(4)).reshape(4, -1).int().contiguous()
    a = ops.paged_decode_gqa(q, kc, vc, bt64.cuda(), n, 0.1)
    b = ops.paged_decode_gqa(q, kc.view(-1, 16, 2, 128), vc.view(-1, 16, 2, 128), bt16.cuda(), n, 0.1)
    ops.check_status()
    assert torch.equal(a, b)


# --------------------------------------------------------------------------------------------- latent rows
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("H,r,dr", [(16, 512, 0), (32, 256, 0), (20, 512, 64), (3, 256, 64), (4, 96, 0), (5, 640, 0), (2, 17, 0)])
def test_latent_decode(H, r, dr, bs, dtype):
    from llm_from_scratch_b200 import ops
    g = gen(r)
    lens = [1, 16, 0, 65, 1500, 333, 64]
    bt, nb = tables(lens, bs)
    lat = torch.randn(nb, bs, r + dr, generator=g).to(dtype)
    q = (torch.randn(len(lens), H, r + dr, generator=g)).to(dtype)
    rope = q[:, :, r:].contiguous().cuda() if dr else None
    got = ops.mla_decode(q[:, :, :r].contiguous().cuda(), rope, lat.cuda(), bt.cuda(), torch.tensor(lens).cuda(), (r + dr) ** -0.5)
    ops.check_status()
    for i, n in enumerate(lens):
        if n == 0:
            assert not got[i].any()
            continue
        c = rows_of(lat, bt, i, n).double()
        want = orc.causal_attention(q[i:i + 1].double(), c[:, None], c[:, None, :r], (r + dr) ** -0.5, None, n - 1)
        assert (got[i].double().cpu() - want[0]).abs().max() <= TOL[dtype] * 2, (i, n)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("r", [96, 512, 50, 7])
def test_latent_rows_in_and_out_of_the_pool(r, dtype):
    from llm_from_scratch_b200 import ops
    g, bs = gen(r), 16
    lens = [33, 1, 16, 50]
    bt, nb = tables(lens, bs)
    T, w = sum(lens), torch.rand(r, generator=g) + 0.5
    proj = torch.randn(T, r + 24 - r % 8, generator=g).to(dtype)
    slots = torch.tensor([int(bt[i, j // bs]) * bs + j % bs for i, n in enumerate(lens) for j in range(n)])
    pool = torch.zeros(nb, bs, r, dtype=dtype, device="cuda")
    rows = ops.latent_norm_store(proj.cuda()[:, 8:8 + r], w.cuda(), 1e-5, pool, slots.cuda())
    close(rows, orc.rms_norm(proj[:, 8:8 + r].double(), w.double(), 1e-5), TOL[dtype])
    back = ops.gather_rows(pool, bt.cuda(), cu(lens).cuda(), max(lens), T)
    assert torch.equal(back, rows)
    part = ops.gather_rows(pool, bt[1:].cuda(), cu(lens)[1:].cuda(), max(lens), T - lens[0])      # offsets that start later
    assert torch.equal(part, rows[lens[0]:])
    ops.check_status()


# ------------------------------------------------------------------------------------------- element-wise
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [64, 37])
def test_gates_activations_and_cap(W, dtype):
    from llm_from_scratch_b200 import ops
    g = gen(W)
    o, proj = 4 * torch.randn(9, W, generator=g), (20 * torch.randn(9, W + 16, generator=g)).to(dtype)
    o = o.to(dtype)
    close(ops.sigmoid_gate(o.cuda(), proj.cuda()[:, 8:8 + W]), o.double() * torch.sigmoid(proj[:, 8:8 + W].double()), TOL[dtype])
    close(ops.squared_relu(o.cuda()), orc.squared_relu(o.double()), TOL[dtype])
    z = 50 * torch.randn(3, W, generator=g)
    close(ops.softcap_logits(z.cuda(), 0.5, 15.0), 15 * torch.tanh(z.double() * 0.5 / 15), 1e-5)
    close(ops.softcap_logits(z.cuda(), 0.5, 0.0), z.double() * 0.5, 1e-6)


# -------------------------------------------------------------------------------------- gated delta rule
class Delta:
    """Random layer: projections of whole sequences, the restatement's outputs and state, and the product's pools."""

    def __init__(self, H, G, dk, dv, taps, lens, dtype, seed=0, slow=False, scale=1.0):
        from llm_from_scratch_b200 import ops
        g = gen(seed)
        up = lambda n: (n + 7) // 8 * 8
        self.sizes = [G * dk, G * dk, H * dv]
        cols = [0, up(G * dk), 2 * up(G * dk)]
        width = cols[2] + up(H * dv)
        self.at = dict(g=width, b=width + up(H * dv), a=width + up(H * dv) + up(H))
        total = self.at["a"] + up(H)
        self.dims, self.lens = (H, G, dk, dv, taps), lens
        self.proj = [(scale * torch.randn(n, total, generator=g)).to(dtype) for n in lens]
        conv = torch.zeros(taps, width)
        for c, n in zip(cols, self.sizes):
            conv[:, c:c + n] = torch.randn(taps, n, generator=g)
        dt, al = torch.randn(H, generator=g), torch.randn(H, generator=g) - (4.0 if slow else 0.5)
        nw = torch.rand(dv, generator=g) + 0.5
        self.c = ops.DeltaRule(H, G, dk, dv, tuple(cols), conv.cuda(), dt.cuda(), al.cuda(), nw.cuda(), 1e-5)
        self.slots = torch.randperm(len(lens) + 2, generator=g)[:len(lens)]
        self.state = torch.full((len(lens) + 2, H, dk, dv), 1e3, device="cuda")      # slots hold what others left
        self.ring = torch.full((len(lens) + 2, taps, width), 1e3, device="cuda")
        self.want, self.final = [], []
        for p in self.proj:
            x = p.double()
            act = [orc.silu(orc.short_conv(x[:, c:c + n], conv[:, c:c + n].t().double())).to(dtype).double()
                   for c, n in zip(cols, self.sizes)]
            n = x.shape[0]
            q, k = orc.unit(act[0].view(n, G, dk)) * dk ** -0.5, orc.unit(act[1].view(n, G, dk))
            o, S = orc.delta_rule(q, k, act[2].view(n, H, dv), torch.sigmoid(self.part(x, "b")),
                                  orc.log_decay(self.part(x, "a"), dt.double(), al.double()))
            o = orc.rms_norm(o, nw.double(), 1e-5).reshape(n, -1) * orc.silu(self.part(x, "g"))
            self.want.append(o)
            self.final.append(S)

    def part(self, x, name):
        H, _, _, dv, _ = self.dims
        return x[:, self.at[name]:self.at[name] + (H * dv if name == "g" else H)]

    def step(self, ranges, general=False):
        """ranges: (sequence, from, to); returns the outputs of each."""
        from llm_from_scratch_b200 import ops
        x = torch.cat([self.proj[s][a:b] for s, a, b in ranges]).cuda()
        slots = self.slots[[s for s, _, _ in ranges]].cuda()
        b, a, g = (self.part(x, n) for n in "bag")
        if all(hi - lo == 1 for _, lo, hi in ranges):
            lens = torch.tensor([hi for _, _, hi in ranges]).cuda()
            y = ops.delta_step(self.c, x, b, a, g, self.state, self.ring, slots, lens)
        else:
            cq = cu([hi - lo for _, lo, hi in ranges]).cuda()
            ck = cu([hi for _, _, hi in ranges]).cuda()
            y = ops.delta_rule(self.c, x, b, a, g, self.state, self.ring, slots, cq, ck, general=general)
        ops.check_status()
        return y.cpu().split([hi - lo for _, lo, hi in ranges])


DELTA_SHAPES = [(4, 2, 64, 64, 4), (2, 2, 128, 128, 4), (2, 1, 128, 64, 4), (3, 1, 64, 128, 2), (3, 1, 48, 32, 2), (6, 2, 32, 112, 3),
                (2, 1, 80, 16, 5), (3, 3, 20, 12, 1), (2, 1, 33, 7, 4), (1, 1, 256, 256, 4), (1, 1, 16, 16, 4)]
STATE_TOL = {torch.float32: 3e-5, torch.bfloat16: 3e-5}      # behind equal activations the state is fp32 in either dtype


def delta_tol(dtype):
    return 1e-4 if dtype == torch.float32 else 2e-2


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", DELTA_SHAPES)
@pytest.mark.parametrize("general", [False, True])
def test_delta_rule_of_whole_prompts(shape, general, dtype):
    d = Delta(*shape, [200, 1, 64, 65, 2, 130], dtype, seed=shape[2])
    got = d.step([(i, 0, n) for i, n in enumerate(d.lens)], general)
    for i, y in enumerate(got):
        close(y, d.want[i], delta_tol(dtype))
        close(d.state[d.slots[i]], d.final[i], 1e-4 if dtype == torch.float32 else 3e-2)
    untouched = [s for s in range(len(d.lens) + 2) if s not in d.slots.tolist()]
    assert (d.state[untouched] == 1e3).all() and (d.ring[untouched] == 1e3).all()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shape", DELTA_SHAPES)
def test_delta_rule_in_portions_and_single_tokens(shape, dtype):
    """Cuts inside chunks and inside the convolution's reach, portions of two tokens, single tokens between portions, and
    unequal sequences beside each other."""
    d = Delta(*shape, [150, 90], dtype, seed=5)
    cuts = [[0, 3, 5, 6, 70, 134, 135, 136, 138, 150], [0, 1, 2, 4, 33, 34, 70, 71, 80, 90]]
    for i in range(9):
        ranges = [(s, cuts[s][i], cuts[s][i + 1]) for s in range(2)]
        if len({b - a == 1 for _, a, b in ranges}) == 2:
            parts = [[r] for r in ranges]            # a step kernel call and a portion call, as in a mixed step
        else:
            parts = [ranges]
        for p in parts:
            for (s, a, b), y in zip(p, d.step(p)):
                close(y, d.want[s][a:b], delta_tol(dtype) * 1.5)


@pytest.mark.parametrize("slow", [True, False])
def test_chunked_delta_rule_keeps_fp32_accuracy(slow):
    """Same bf16 activations for both kernels: the chunked tensor-core form and the fp32 token-by-token form agree far
    below bf16 resolution, in the state and through 400 tokens."""
    d = Delta(2, 1, 128, 64, 4, [400], torch.bfloat16, seed=9, slow=slow)
    e = Delta(2, 1, 128, 64, 4, [400], torch.bfloat16, seed=9, slow=slow)
    y = d.step([(0, 0, 400)])[0]
    z = e.step([(0, 0, 400)], general=True)[0]
    close(d.state[d.slots[0]], e.state[e.slots[0]].cpu(), STATE_TOL[torch.bfloat16])
    assert (y.float() != z.float()).float().mean() < 0.01            # outputs differ in a bf16 rounding here and there


def test_delta_rule_with_strong_decays_and_large_inputs():
    d = Delta(4, 2, 64, 64, 4, [130, 64], torch.bfloat16, seed=2, scale=12.0)
    for y, w in zip(d.step([(0, 0, 130), (1, 0, 64)]), d.want):
        assert torch.isfinite(y.float()).all()
        close(y, w, 8e-2)


def test_equal_keys_in_a_chunk():
    """Every token writes under the same key with full strength: the triangular solve is at its hardest, and reading
    returns the last value only."""
    from llm_from_scratch_b200 import ops
    H, dk, dv, n = 1, 64, 64, 128
    width = 2 * dk + dv
    conv = torch.ones(1, width)
    c = ops.DeltaRule(H, 1, dk, dv, (0, dk, 2 * dk), conv.cuda(), torch.zeros(1).cuda(), torch.full((1,), -30.0).cuda(),
                      torch.ones(dv).cuda(), 1e-5)
    g = gen(0)
    x = torch.zeros(n, width + dv + 16)
    x[:, :2 * dk] = torch.randn(dk, generator=g).repeat(2) + 1.0
    x[:, 2 * dk:width] = torch.randn(n, dv, generator=g)
    x[:, width:width + dv] = 1.0
    x[:, width + dv] = 40.0                     # beta = 1
    x = x.bfloat16()
    state, ring = torch.zeros(1, H, dk, dv, device="cuda"), torch.zeros(1, 1, width, device="cuda")
    xc = x.cuda()
    y = ops.delta_rule(c, xc, xc[:, width + dv:width + dv + 1], xc[:, width + dv + 8:width + dv + 9], xc[:, width:width + dv],
                       state, ring, torch.zeros(1, dtype=torch.int64).cuda(), cu([n]).cuda(), cu([n]).cuda())
    v = orc.silu(x[:, 2 * dk:width].double()).bfloat16().double()
    close(y, orc.rms(v * dk ** -0.5, 1e-5) * orc.silu(torch.tensor(1.0, dtype=torch.float64)), 3e-2)
    ops.check_status()


def test_rows_of_no_sequence_are_left_alone():
    """Padding tokens behind the last sequence, skipped slots and empty contexts change nothing."""
    from llm_from_scratch_b200 import ops
    d = Delta(2, 1, 64, 32, 4, [70, 5], torch.bfloat16, seed=4)
    x = torch.cat(d.proj + [torch.full((13, d.proj[0].shape[1]), float("nan")).bfloat16()]).cuda()
    b, a, g = (d.part(x, n) for n in "bag")
    slots = d.slots.clone().cuda()
    slots[1] = -1
    before = d.state.clone()
    c = cu([70, 5]).cuda()
    y = ops.delta_rule(d.c, x, b, a, g, d.state, d.ring, slots, c, c)
    close(y[:70], d.want[0], 4e-2)
    keep = [s for s in range(4) if s != int(d.slots[0])]
    assert torch.equal(d.state[keep], before[keep])
    lens = torch.tensor([0, 71]).cuda()
    before = d.state.clone()
    ops.delta_step(d.c, x, b, a, g, d.state, d.ring, torch.stack([slots[0], slots[1]]), lens)
    ops.check_status()
    assert torch.equal(d.state, before)
