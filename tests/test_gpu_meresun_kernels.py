"""Kernels behind the Meresun family, each alone, against the plain CPU restatement."""
import pytest
import torch

from oracle import meresun as orc

pytestmark = pytest.mark.gpu
DTYPES = [torch.float32, torch.bfloat16]
TOL = {torch.float32: 3e-5, torch.bfloat16: 2e-2}
YARN = dict(factor=8.0, original=256, fast=16.0, slow=1.0)


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


def slots_of(bt, i, n, bs):
    return torch.tensor([int(bt[i, j // bs]) * bs + j % bs for j in range(n)], dtype=torch.int64)


def rotation(base, dims, scaling=None):
    from llm_from_scratch_b200 import ops
    return ops.Rotation(base, dims, "cuda", ops.YarnScaling(**scaling) if scaling else None)


# ------------------------------------------------------------------------------------ residual boundaries
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,groups", [(64, 1), (64, 4), (100, 5), (99, 3), (333, 1), (1024, 2), (4096, 8), (6144, 3), (6144, 128),
                                      (10000, 4), (70, 35)])
def test_residual_group_norm(d, groups, dtype):
    from llm_from_scratch_b200 import ops
    T, eps, g = 7, 1e-4, gen(d + groups)
    embed = torch.randn(50, d, generator=g).to(dtype)
    toks = torch.randint(0, 50, (T,), generator=g)
    y = (3 * torch.randn(T, d, generator=g)).to(dtype)
    w, nw = torch.rand(d, generator=g) + 0.5, torch.rand(d, generator=g) + 0.5
    part_size = torch.logspace(-1, 1, groups).repeat_interleave(d // groups)          # parts of unlike size
    e = embed[toks].double() * 0.3
    emb = dict(tokens=toks.cuda(), embed=embed.cuda(), embed_scale=0.3)
    x = torch.full((T, d), 7.0, device="cuda")
    h = ops.residual_group_norm(x, nw.cuda(), groups, eps, dtype, start=True, **emb)
    close(x, e, 1e-6)
    close(h, orc.group_norm(e, nw.double(), groups, eps), TOL[dtype])
    x.copy_((torch.randn(T, d, generator=g) * part_size).cuda())
    for kw, use_y, use_e in ((dict(y=y.cuda(), y_norm_w=w.cuda()), 1, 0), (dict(y=y.cuda(), y_norm_w=w.cuda(), **emb), 1, 1), (emb, 0, 1)):
        want = x.cpu().double() + use_y * orc.rms_norm(y.double(), w.double(), eps) + use_e * e
        h = ops.residual_group_norm(x, nw.cuda(), groups, eps, dtype, **kw)
        close(x, want, 1e-5)
        close(h, orc.group_norm(want, nw.double(), groups, eps), TOL[dtype])
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,d,top", [(5, 64, 3), (9, 37, 1), (130, 256, 8), (3, 4096, 2), (1, 24, 4)])
def test_gated_residual(T, d, top, dtype):
    from llm_from_scratch_b200 import ops
    g = gen(d)
    up = (d + 7) // 8 * 8
    proj = (3 * torch.randn(T, 16 + 2 * up, generator=g)).to(dtype)
    y1, y2 = (torch.randn(T, d, generator=g).to(dtype) for _ in range(2))
    rows, w = torch.randn(T * top, d, generator=g).to(dtype), torch.rand(T, top, generator=g)
    slot = torch.randperm(T * top, generator=g).view(T, top).int()
    x0 = torch.randn(T, d, generator=g)
    pc = proj.cuda()
    g1, g2 = pc[:, 16:16 + d], pc[:, 16 + up:16 + up + d]
    s1, s2 = torch.sigmoid(g1.cpu().double()), torch.sigmoid(g2.cpu().double())
    one = x0.double() + y1.double() * s1
    mixture = (rows.double()[slot.long()] * w.double()[:, :, None]).sum(1)
    for args, want in (((), one), ((y2.cuda(), g2), one + y2.double() * s2),
                       ((rows.cuda(), g2, w.cuda(), slot.cuda()), one + mixture * s2)):
        x = x0.cuda()
        h = ops.gated_residual(x, y1.cuda(), g1, *args)
        close(x, want, 1e-5)
        assert torch.equal(h, x.to(dtype))
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W", [8, 40, 37, 1000, 2816, 11264, 20000, 40000])
def test_poly_norm(W, dtype):
    from llm_from_scratch_b200 import ops
    g, coef = gen(W), torch.tensor([0.7, -0.4, 0.3, 0.2])
    z = (torch.randn(5, W + 16, generator=g) * torch.tensor([1e-4, 0.1, 1.0, 5.0, 30.0])[:, None]).to(dtype)
    got = ops.poly_norm(z.cuda()[:, 8:8 + W], coef.cuda(), 1e-5)
    want = orc.poly_norm(z[:, 8:8 + W].double(), coef.double(), 1e-5)
    for t in range(5):
        close(got[t], want[t], TOL[dtype])


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("W,first", [(24, 48), (7, 0), (256, 512)])
def test_gelu_of_a_projection_scales_table_rows(W, first, dtype):
    from llm_from_scratch_b200 import ops
    g = gen(W)
    u, table = (3 * torch.randn(11, W, generator=g)).to(dtype), torch.randn(30, first + W + 5, generator=g).to(dtype)
    toks = torch.randint(0, 30, (11,), generator=g)
    want = orc.gelu_tanh(u.double()) * table[toks, first:first + W].double()
    close(ops.gelu_table(u.cuda(), table.cuda(), first, toks.cuda()), want, TOL[dtype])
    ops.check_status()


# ---------------------------------------------------------------------------------- latents, rotation, pool
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rq,r,dr,dims,scaling", [(40, 48, 8, 8, YARN), (512, 512, 64, 64, YARN), (33, 17, 6, 4, None), (80, 64, 0, 0, None),
                                                  (24, 40, 70, 70, YARN), (7, 9, 5, 2, None)])
def test_latent_prologue(rq, r, dr, dims, scaling, dtype):
    from llm_from_scratch_b200 import ops
    g, T, bs = gen(rq), 11, 16
    proj = (2 * torch.randn(T, 200 + rq + r + dr, generator=g)).to(dtype)
    off = 8 + (rq + 7) // 8 * 8
    dq, dkv = proj[:, 8:8 + rq], proj[:, off:off + r + dr]
    wq, wk = torch.rand(rq, generator=g) + 0.5, torch.rand(r, generator=g) + 0.5
    pos = torch.tensor([0, 1, 2, 63, 64, 1000, 4095, 70001, 1 << 20, 5, 6])
    slots = torch.tensor([3, -1, 17, 16, 40, 5, 6, 7, 8, 9, 31])
    pool = torch.zeros(3, bs, r + dr, dtype=dtype, device="cuda")
    pc = proj.cuda()
    q, rows = ops.latent_prologue(pc[:, 8:8 + rq], wq.cuda(), pc[:, off:off + r + dr], wk.cuda(), 1e-5, rotation(500.0, dims, scaling),
                                  pos.cuda(), pool, slots.cuda())
    ops.check_status()
    close(q, orc.rms_norm(dq.double(), wq.double(), 1e-5), TOL[dtype])
    close(rows[:, :r], orc.rms_norm(dkv[:, :r].double(), wk.double(), 1e-5), TOL[dtype])
    if dr:
        want = torch.cat([orc.rotate_pairs(dkv[t:t + 1, None, r:].double(), dims, 500.0, scaling, int(pos[t])) for t in range(T)])
        close(rows[:, r:], want[:, 0], TOL[dtype])
    flat = pool.view(-1, r + dr)
    for t in range(T):
        if slots[t] >= 0:
            assert torch.equal(flat[slots[t]], rows[t])
    rest = [i for i in range(3 * bs) if i not in set(slots.tolist())]
    assert not flat[rest].any()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,D,dr,dims,scaling", [(3, 32, 8, 8, YARN), (16, 192, 64, 64, YARN), (2, 15, 5, 4, None), (1, 2, 2, 2, None),
                                                 (5, 40, 40, 40, YARN)])
def test_rotate_heads(H, D, dr, dims, scaling, dtype):
    from llm_from_scratch_b200 import ops
    g = gen(D)
    q = torch.randn(9, H, D, generator=g).to(dtype)
    pos = torch.tensor([0, 1, 5, 77, 1 << 18, 3, 4, 2000, 9])
    qc = q.cuda()
    tail = ops.rotate_heads(qc, dr, rotation(1000.0, dims, scaling), pos.cuda(), 4)
    turned = torch.cat([orc.rotate_pairs(q[t:t + 1, :, D - dr:].double(), dims, 1000.0, scaling, int(pos[t])) for t in range(9)])
    close(qc, torch.cat([q[..., :D - dr].double(), turned], -1), TOL[dtype])
    assert torch.equal(qc[..., :D - dr].cpu(), q[..., :D - dr]) and torch.equal(tail, qc[:4, :, D - dr:])
    assert ops.rotate_heads(qc, dr, rotation(1000.0, dims, scaling), pos.cuda()) is None


@pytest.mark.parametrize("W", [56, 9])
def test_gather_the_ends_of_contexts(W):
    from llm_from_scratch_b200 import ops
    bs, lens, ends = 16, [33, 1, 16, 50, 64], [7, 1, 16, 35, 17]
    bt, nb = tables(lens, bs)
    pool = torch.randn(nb, bs, W, generator=gen(W)).bfloat16()
    flat = pool.view(-1, W)
    want = torch.cat([flat[slots_of(bt, i, n, bs)[n - e:]] for i, (n, e) in enumerate(zip(lens, ends))])
    got = ops.gather_rows(pool.cuda(), bt.cuda(), cu(ends).cuda(), max(ends), sum(ends), cu(lens).cuda())
    ops.check_status()
    assert torch.equal(got.cpu(), want)
    torch.full((192, W), float("nan"), device="cuda")                  # what freed memory may hold
    got = ops.gather_rows(pool.cuda(), bt.cuda(), cu(ends).cuda(), max(ends), sum(ends), cu(lens).cuda(), 64).cpu()
    assert got.shape == (128, W) and torch.equal(got[:sum(ends)], want) and not got[sum(ends):].any()


# ------------------------------------------------------------------------------------- windowed attention
def ramp(k, q, sharp):
    """Two channels that make a key's score fall by ``sharp`` per position, exactly in bf16: the oldest key a query sees takes
    nearly all of its weight, so a window that is off by one token gives another result altogether.  k [nk, ., D], q [nq, ., D]."""
    j = torch.arange(k.shape[0])
    k[..., 0], k[..., 1] = -(j % 64).to(k.dtype)[:, None], -(j // 64).to(k.dtype)[:, None]
    q[..., 0], q[..., 1] = sharp, 64 * sharp


SHAPES = [(4, 4, 192, 64, 128), (3, 3, 192, 0, 128), (4, 2, 128, 0, 128), (3, 3, 40, 16, 40), (2, 2, 80, 16, 88), (6, 3, 64, 0, 64),
          (2, 2, 136, 72, 24), (3, 3, 33, 9, 21), (2, 2, 300, 20, 140), (1, 1, 16, 8, 8)]
WINDOWS = [0, 1, 2, 63, 64, 65, 100, 257]


def windowed_case(Hq, G, Dqk, Dv, qlens, klens, dtype, seed, sharp):
    g = gen(seed)
    q = [torch.randn(n, Hq, Dqk, generator=g).to(dtype) for n in qlens]
    k = [torch.randn(n, G, Dqk, generator=g).to(dtype) for n in klens]
    v = [torch.randn(n, G, Dv, generator=g).to(dtype) for n in klens]
    if sharp:
        for a, b in zip(k, q):
            ramp(a, b, sharp)
    return q, k, v


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("Hq,G,Dqk,tail,Dv", SHAPES)
def test_windowed_prefill(Hq, G, Dqk, tail, Dv, dtype):
    """Windows from one token to wider than the context, contexts that begin before the portion, tile borders; with and
    without a tile list; the key's shared part is the same for all heads."""
    from llm_from_scratch_b200 import ops
    scale, qlens = 0.25, [1, 70, 2, 300]
    klens = [n + e for n, e in zip(qlens, (5, 0, 200, 64))]
    sink = torch.randn(Hq, generator=gen(1))
    cq, ck = cu(qlens).cuda(), cu(klens).cuda()
    for window in WINDOWS:
        for sharp in (0.0, 4.0):
            q, k, v = windowed_case(Hq, G, Dqk, Dv, qlens, klens, dtype, Dqk + window, sharp)
            if tail:
                for x in k:
                    x[..., Dqk - tail:] = x[:, :1, Dqk - tail:]
            of = torch.arange(Hq) // (Hq // G)
            want = torch.cat([orc.windowed_attention(a.double(), b.double()[:, of], c.double()[:, of], scale, sink.double(), window,
                                                     len(b) - len(a)) for a, b, c in zip(q, k, v)])
            kc, vc, qc = torch.cat(k).cuda(), torch.cat(v).cuda(), torch.cat(q).cuda()
            head, rest = kc[..., :Dqk - tail].contiguous(), kc[:, 0, Dqk - tail:].contiguous() if tail else None
            for rows in (0, ops.prefill_window_tile_rows(Hq, G, Dqk, tail, Dv, dtype)):
                plan = ops.prefill_plan(cq, sum(qlens), max(qlens), rows)
                got = ops.prefill_varlen_window(qc, head, rest, vc, cq, ck, max(qlens), scale, window, sink.cuda(), plan=plan)
                ops.check_status()
                assert (got.double().cpu() - want).abs().max() <= TOL[dtype] * (1 if dtype == torch.float32 else 1.5), (window, sharp)


def test_windowed_prefill_without_a_window_is_the_plain_one():
    from llm_from_scratch_b200 import ops
    g, lens = gen(4), [300, 64, 1]
    q, k, v = (torch.randn(sum(lens), 4, 128, generator=g).bfloat16().cuda() for _ in range(3))
    c = cu(lens).cuda()
    a = ops.prefill_varlen(q, k, v, c, c, 300, 300, 0.1)
    b = ops.prefill_varlen_window(q, k, None, v, c, c, 300, 0.1)
    assert torch.equal(a, b)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [16, 64])
@pytest.mark.parametrize("H,r,dr", [(16, 512, 64), (20, 512, 64), (5, 512, 0), (3, 256, 64), (33, 256, 0), (6, 48, 8), (2, 17, 5)])
def test_windowed_latent_decode(H, r, dr, bs, dtype):
    """Contexts at block and window borders, cut over many CTAs; tokens just inside and just outside the window decide."""
    from llm_from_scratch_b200 import ops
    g, scale = gen(r + bs), 0.25
    lens = [1, 16, 0, 65, 1500, 333, 64, 100, 101, 163]
    bt, nb = tables(lens, bs)
    lat = torch.randn(nb, bs, r + dr, generator=g).to(dtype)
    sink = torch.randn(H, generator=g)
    q = torch.randn(len(lens), H, r + dr, generator=g).to(dtype)
    flat = lat.view(-1, r + dr)
    for sharp in (0.0, 4.0):
        if sharp:
            q[..., 0], q[..., 1] = sharp, 64 * sharp
            for i, n in enumerate(lens):
                j, at = torch.arange(n), slots_of(bt, i, n, bs)
                flat[at, 0], flat[at, 1] = -(j % 64).to(dtype), -(j // 64).to(dtype)
        for window in (0, 1, 15, 16, 17, 64, 100, 1000):
            rope = q[:, :, r:].contiguous().cuda() if dr else None
            got = ops.mla_decode(q[:, :, :r].contiguous().cuda(), rope, lat.cuda(), bt.cuda(), torch.tensor(lens).cuda(), scale,
                                 window=window, sink=sink.cuda())
            ops.check_status()
            for i, n in enumerate(lens):
                if n == 0:
                    assert not got[i].any()
                    continue
                c = flat[slots_of(bt, i, n, bs)].double()[:, None].expand(n, H, r + dr)
                want = orc.windowed_attention(q[i:i + 1].double(), c, c[..., :r], scale, sink.double(), window, n - 1)
                close(got[i], want[0], TOL[dtype] * 2)


def test_latent_decode_with_a_sink_that_takes_everything():
    from llm_from_scratch_b200 import ops
    g = gen(0)
    bt, nb = tables([200], 16)
    lat, q = torch.randn(nb, 16, 576, generator=g).bfloat16().cuda(), torch.randn(1, 16, 576, generator=g).bfloat16().cuda()
    sink = torch.full((16,), -300.0)
    sink[3] = 300.0
    args = (q[..., :512].contiguous(), q[..., 512:].contiguous(), lat, bt.cuda(), torch.tensor([200]).cuda(), 0.05)
    with_sink, plain = ops.mla_decode(*args, sink=sink.cuda()), ops.mla_decode(*args)
    assert not with_sink[0, 3].any()
    close(with_sink[0, 4:], plain[0, 4:].cpu(), 1e-2)


# -------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T", [1, 7, 128, 129, 2500])
@pytest.mark.parametrize("E,top,groups,keep", [(12, 3, 3, 2), (16, 2, 1, 1), (64, 8, 8, 4), (256, 8, 8, 4), (300, 6, 10, 3), (5, 5, 1, 1),
                                               (6, 1, 6, 2), (40, 4, 2, 1)])
def test_group_route(E, top, groups, keep, T):
    from llm_from_scratch_b200 import ops
    g = gen(E + T)
    z, corr = 2 * torch.randn(T, E, generator=g), torch.randn(E, generator=g) - 1.0           # choice scores of both signs
    tok, w, offs, slot = (t.cpu() for t in ops.moe_group_route(z.cuda(), corr.cuda(), top, groups, keep))
    n = min(T, 150)
    ends = offs.long()
    expert_of = torch.bucketize(slot.long(), ends, right=True)                                # [T, top]
    for t, (chosen, wts, _) in enumerate(orc.route(z[:n].double(), torch.eye(E).double(), corr.double(), groups, keep, top)):
        assert sorted(expert_of[t].tolist()) == chosen
        order = expert_of[t].argsort()
        assert torch.allclose(w[t][order].double(), wts, rtol=1e-5)
    # rows grouped by expert, every (token, choice) in one of them
    assert int(offs[-1]) == T * top and sorted(slot.reshape(-1).tolist()) == list(range(T * top))
    assert torch.equal(tok[slot.long()], torch.arange(T).int()[:, None].expand(T, top))
    assert (expert_of.sort(1).values.diff(dim=1) > 0).all()


@pytest.mark.parametrize("glu", [False, True])
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("counts,k,n", [([5, 0, 17, 1], 120, 40), ([130, 0, 3], 64, 200), ([400, 300], 256, 384), ([9, 70, 0, 0, 2], 33, 21),
                                        ([0, 0, 1], 8, 8), ([90, 1, 200], 100, 36)])
def test_grouped_linear(counts, k, n, dtype, glu):
    from llm_from_scratch_b200 import ops
    g, E, R = gen(k + n), len(counts), sum(counts)
    x = torch.randn(R, k, generator=g).to(dtype)
    w = (2 * torch.randn(E, 2 * n if glu else n, k, generator=g) * k ** -0.5).to(dtype)
    offs = torch.tensor(counts).cumsum(0).int()
    rows = []
    for e, part in enumerate(x.double().split(counts)):
        y = part @ w[e].double().T
        rows.append(orc.clamped_glu(y[:, :n], y[:, n:], 1.1) if glu else y)
    got = ops.moe_grouped_linear(x.cuda(), w.cuda(), offs.cuda(), glu=(1.1, 1.702) if glu else None)
    ops.check_status()
    close(got, torch.cat(rows), TOL[dtype])
