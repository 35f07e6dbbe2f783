"""Kernels behind the Sodonex family, each alone, against the plain CPU restatement."""
import pytest
import torch

from oracle import sodonex as orc

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


def slots_of(bt, i, n, bs):
    return torch.tensor([int(bt[i, j // bs]) * bs + j % bs for j in range(n)], dtype=torch.int64)


def ragged(q, k, slots):
    """Rows of a step: portions of q tokens at the ends of contexts of k."""
    from llm_from_scratch_b200 import ops
    return ops.StepRows(torch.tensor(slots).cuda(), cu(q).cuda(), cu(k).cuda())


def singles(lens, slots):
    from llm_from_scratch_b200 import ops
    return ops.StepRows(torch.tensor(slots).cuda(), context_lens=torch.tensor(lens).cuda())


# ------------------------------------------------------------------------------------ residual boundaries
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d", [8, 64, 100, 99, 1000, 1024, 4096, 6144, 10000])
def test_residual_with_one_number_per_norm(d, dtype):
    from llm_from_scratch_b200 import ops
    T, eps, g = 9, 1e-3, gen(d)
    embed, toks = torch.randn(50, d, generator=g).to(dtype), torch.randint(0, 50, (T,), generator=g)
    y = (torch.randn(T, d, generator=g) * torch.logspace(-2, 1, T)[:, None]).to(dtype)
    x = torch.empty(T, d, device="cuda")
    h = ops.shift_residual(None, eps, dtype, x_out=x, tokens=toks.cuda(), embed=embed.cuda(), embed_scale=0.3)
    want = embed[toks].double() * 0.3
    close(x, want, 1e-6)
    assert torch.equal(h, x.to(dtype))
    want = x.cpu().double() + orc.gain_norm(y.double(), torch.tensor(-0.7).double(), eps)
    h = ops.shift_residual(x, eps, dtype, x_out=x, y=y.cuda(), gain=-0.7)
    close(x, want, 1e-5)
    assert torch.equal(h, x.to(dtype))
    before, want = x.clone(), x.cpu().double() + orc.gain_norm(y.double(), torch.tensor(0.4).double(), eps)
    h = ops.shift_residual(x, eps, dtype, y=y.cuda(), gain=0.4, final_gain=1.3)
    close(h, orc.gain_norm(want, torch.tensor(1.3).double(), eps), TOL[dtype])
    assert torch.equal(x, before)                                    # nothing was asked to be written
    ops.check_status()


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("T,d,top", [(5, 64, 3), (9, 37, 1), (130, 256, 8), (3, 4096, 2), (2100, 72, 4)])
def test_residual_sums_a_tokens_experts(T, d, top, dtype):
    from llm_from_scratch_b200 import ops
    g = gen(d)
    rows, wts = torch.randn(T * top, d, generator=g).to(dtype), torch.rand(T, top, generator=g)
    slot = torch.randperm(T * top, generator=g).view(T, top).int()
    x0 = torch.randn(T, d, generator=g)
    mixture = (rows.double()[slot.long()] * wts.double()[:, :, None]).sum(1)
    want = x0.double() + orc.gain_norm(mixture, torch.tensor(0.9).double(), 1e-5)
    x = x0.cuda()
    h = ops.shift_residual(x, 1e-5, dtype, x_out=x, y=rows.cuda(), gain=0.9, row_weight=wts.cuda(), slot_to_row=slot.cuda())
    ops.check_status()
    close(x, want, 1e-5)
    assert torch.equal(h, x.to(dtype))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("d,sizes", [(64, [1, 2, 3, 4, 5, 9]), (100, [7, 1, 30, 2]), (99, [4, 8, 1]), (2048, [5, 2, 1, 16]),
                                     (6144, [3, 1, 6]), (64, [2040, 3, 90]), (4096, [2050, 2])])
def test_shift_carries_the_last_token_from_step_to_step(d, sizes, dtype):
    """Three sequences in portions of unlike sizes beside each other, with padding rows behind them, then one token each, then
    new sequences in the slots of the old ones: the mixed rows are those of each sequence in one piece."""
    from llm_from_scratch_b200 import ops
    g, eps, shift = gen(d), 1e-5, torch.rand(d, generator=gen(1))
    n = sum(sizes) + 1
    state = torch.full((5, d), float("nan"), device="cuda")
    for turn in range(2):
        x0 = [torch.randn(n, d, generator=g) for _ in range(3)]
        y0 = [torch.randn(n, d, generator=g).to(dtype) for _ in range(3)]
        full = [x.double() + orc.gain_norm(y.double(), torch.tensor(0.6).double(), eps) for x, y in zip(x0, y0)]
        want = [orc.token_shift(x, shift.double()) for x in full]
        at, slots = [0, 0, 0], [4, 0, 2] if turn else [1, 2, 4]
        orders = [sizes, sizes[::-1], sizes[1:] + sizes[:1]]
        for i in range(len(sizes)):
            take = [orders[s][i] for s in range(3)]
            cat = lambda parts: torch.cat([p[a:a + t] for p, a, t in zip(parts, at, take)])
            pad = 5
            x, y = (torch.cat([cat(z), torch.ones(pad, d, dtype=z[0].dtype)]).cuda() for z in (x0, y0))
            out = torch.empty_like(x)
            h = ops.shift_residual(x, eps, dtype, x_out=out, y=y, gain=0.6, shift=shift.cuda(), state=state,
                                   rows=ragged(take, [a + t for a, t in zip(at, take)], slots))
            ops.check_status()
            close(out[:-pad], cat(full), 1e-5)
            close(h[:-pad], cat(want), TOL[dtype])
            assert torch.isfinite(h[-pad:]).all()
            at = [a + t for a, t in zip(at, take)]
            close(state[slots], torch.stack([f[a - 1] for f, a in zip(full, at)]), 1e-5)
        x, y = (torch.cat([z[s][-1:] for s in (0, 1, 2)] + [torch.ones(1, d, dtype=z[0].dtype)]).cuda() for z in (x0, y0))
        h = ops.shift_residual(x, eps, dtype, x_out=torch.empty_like(x), y=y, gain=0.6, shift=shift.cuda(), state=state,
                               rows=singles([n, n, n, 0], slots + [-1]))
        ops.check_status()
        close(h[:3], torch.stack([z[-1] for z in want]), TOL[dtype])
        close(state[slots], torch.stack([f[-1] for f in full]), 1e-5)


def test_shift_of_the_embedding_starts_from_zeros():
    from llm_from_scratch_b200 import ops
    embed, toks, shift = torch.randn(20, 48, generator=gen(1)), torch.tensor([3, 4, 5, 3, 9]), torch.rand(48, generator=gen(2))
    state, out = torch.full((2, 48), 7.0, device="cuda"), torch.empty(5, 48, device="cuda")
    h = ops.shift_residual(None, 1e-5, torch.float32, x_out=out, tokens=toks.cuda(), embed=embed.cuda(), embed_scale=2.0,
                           shift=shift.cuda(), state=state, rows=ragged([3, 2], [3, 2], [1, 0]))
    x = 2 * embed[toks].double()
    close(h, torch.cat([orc.token_shift(x[:3], shift.double()), orc.token_shift(x[3:], shift.double())]), 1e-6)
    close(state, x[[4, 2]], 1e-6)
    with pytest.raises(ValueError):
        ops.shift_residual(out, 1e-5, torch.float32, x_out=out, y=h, shift=shift.cuda(), state=state, rows=singles([1] * 5, [0] * 5))


# -------------------------------------------------------------------------- convolution, norm, rotation, pool
SIZES = [(6, 2, 24, 8, 4), (4, 1, 32, 32, 3), (16, 4, 128, 128, 2), (3, 3, 40, 16, 4), (3, 1, 7, 4, 5), (2, 2, 9, 0, 1), (32, 8, 128, 64, 4),
         (1, 1, 8, 2, 20), (48, 8, 128, 32, 3), (2, 1, 300, 100, 3), (8, 8, 16, 16, 1)]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,dims,taps", SIZES)
def test_conv_norm_rope_store(H, G, D, dims, taps, dtype):
    """Two sequences in portions down to one token beside each other, with padding rows, then single tokens; slots are used by a
    second pair of sequences without being cleared."""
    from llm_from_scratch_b200 import ops
    g, eps, base, bs, Cq, Ck = gen(D + taps), 1e-5, 300.0, 16, H * D, G * D
    up = (Cq + 7) // 8 * 8
    wq, wk = (torch.randn(c, taps, generator=g) * taps ** -0.5 for c in (Cq, Ck))
    nq, nk = (torch.rand(c, generator=g) + 0.5 for c in (Cq, Ck))
    freq = ops.rotary_frequencies(base, dims, "cuda")
    ring = torch.full((4, max(taps - 1, 1), Cq + Ck), float("nan"), device="cuda") if taps > 1 else None
    sizes = [[19, 2, 1, 33, 3], [1, 40, 2, 1, 16]]
    n = [sum(s) + 2 for s in sizes]
    for slots in ([3, 0], [0, 1]):
        # neighbouring tokens of very unlike size: a tap that is one off shows
        proj = [(torch.randn(m, up + Ck + 8, generator=g) * (1 + 3 * (torch.arange(m) % 3 == 0))[:, None]).to(dtype) for m in n]
        kc, vc = (torch.zeros(16, bs, G, D, dtype=dtype, device="cuda") for _ in range(2))
        uq, uk = ([orc.short_conv(p[:, a:a + c].double(), w.double()) for p in proj] for a, c, w in ((0, Cq, wq), (up, Ck, wk)))
        rot = lambda u, w, heads: orc.rotate_half(orc.whole_norm(u, w.double(), eps).view(len(u), heads, D), dims, base)
        want = [(rot(a, nq, H), rot(b, nk, G), b.view(len(b), G, D)) for a, b in zip(uq, uk)]
        page = [torch.arange(m) + 100 * s for s, m in enumerate(n)]
        at = [0, 0]

        def step(take, rows, pad, packed):
            cat = lambda parts: torch.cat([p[a:a + t] for p, a, t in zip(parts, at, take)])
            x = torch.cat([cat(proj), torch.ones(pad, up + Ck + 8, dtype=dtype)]).cuda()
            pos = torch.cat([torch.arange(a, a + t) for a, t in zip(at, take)] + [torch.zeros(pad, dtype=torch.int64)])
            where = torch.cat([cat(page), torch.full((pad,), -1)])
            got = ops.conv_norm_rope_store(x[:, :Cq], x[:, up:up + Ck], wq.t().contiguous().cuda(), wk.t().contiguous().cuda(), ring, rows,
                                           nq.cuda(), nk.cuda(), eps, freq, pos.cuda(), kc, vc, where.cuda(), packed=packed)
            ops.check_status()
            for y, i in zip(got, range(3)):
                if y is None:
                    assert not packed and i > 0
                    continue
                assert torch.isfinite(y).all()
                close(y[:len(y) - pad] if pad else y, cat([z[i] for z in want]), TOL[dtype])
            return got

        for i in range(len(sizes[0])):
            take = [s[i] for s in sizes]
            step(take, ragged(take, [a + t for a, t in zip(at, take)], slots), 3 * (i % 2), True)
            at = [a + t for a, t in zip(at, take)]
        for i in range(2):
            step([1, 1], singles([a + 1 for a in at], slots), 0, i == 0)
            at = [a + 1 for a in at]
        for s in range(2):
            for pool, i in ((kc, 1), (vc, 2)):
                close(pool.view(-1, G, D)[page[s].cuda()], want[s][i], TOL[dtype])


@pytest.mark.parametrize("D,dims", [(24, 16), (128, 128), (10, 4)])
def test_rotation_keeps_large_positions(D, dims):
    from llm_from_scratch_b200 import ops
    pos = torch.tensor([0, 1, 63, 4095, 70001, 1 << 20])
    x, one = torch.randn(6, 2 * D, generator=gen(D)), torch.ones(1, D)
    kc, vc = (torch.zeros(1, 16, 1, D, device="cuda") for _ in range(2))
    q, _, _ = ops.conv_norm_rope_store(x.cuda()[:, :D], x.cuda()[:, D:], one.cuda(), one.cuda(), None, singles((pos + 1).tolist(), list(range(6))),
                                       one.cuda(), one.cuda(), 1e-5, ops.rotary_frequencies(5e4, dims, "cuda"), pos.cuda(), kc, vc,
                                       torch.arange(6).cuda())
    u = orc.rms(x[:, None, :D].double(), 1e-5)
    close(q, torch.cat([orc.rotate_half(u[t:t + 1], dims, 5e4, int(pos[t])) for t in range(6)]), 1e-5)


# ------------------------------------------------------------------------------------- sigmoid attention
def edges(v, chunk):
    """Values that are large at the first and last position of every chunk: a chunk that is off by one token shows."""
    if chunk > 1:
        v[::chunk] *= 12.0
        v[chunk - 1::chunk] *= 12.0
    return v


SHAPES = [(4, 2, 128, 128), (3, 3, 128, 128), (8, 2, 64, 64), (2, 1, 64, 64), (3, 1, 40, 40), (6, 3, 96, 96), (2, 2, 136, 24), (3, 3, 33, 33),
          (2, 1, 300, 300), (1, 1, 16, 8)]
CHUNKS = [0, 1, 2, 63, 64, 100, 128, 256, 257]


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("H,G,D,Dv", SHAPES)
def test_sigmoid_attention_of_prompts(H, G, D, Dv, dtype):
    """Chunks from one token to wider than the context, packed contexts that begin a chunk before the portion, tile borders;
    with and without a tile list and a gate."""
    from llm_from_scratch_b200 import ops
    scale, qlens, g = 1.5 * D ** -0.5, [1, 70, 2, 300, 129], gen(D)
    of = torch.arange(H) // (H // G)
    bias, cq = torch.linspace(-2.0, 1.0, H), cu(qlens).cuda()
    gate = (2 * torch.randn(sum(qlens), H + 5, generator=g)).to(dtype)
    for chunk in CHUNKS:
        # a portion that starts in the middle of its chunk has the chunk's keys in front
        extra = [0 if chunk == 1 else min(e, chunk - 1) if chunk else e for e in (5, 0, 200, 64, 127)]
        klens = [n + e for n, e in zip(qlens, extra)]
        q = [torch.randn(n, H, D, generator=g).to(dtype) for n in qlens]
        k = [torch.randn(n, G, D, generator=g).to(dtype) for n in klens]
        v = [edges(torch.randn(n, G, Dv, generator=g), chunk).to(dtype) for n in klens]
        want = torch.cat([orc.sigmoid_attention(a.double(), b.double(), c.double(), scale, bias.double(), chunk, len(b) - len(a))
                          for a, b, c in zip(q, k, v)])
        gated = want * torch.sigmoid(gate[:, 3:3 + H].double())[..., None]
        qc, kc, vc, gc = torch.cat(q).cuda(), torch.cat(k).cuda(), torch.cat(v).cuda(), gate.cuda()
        for rows in {0, ops.sigmoid_attention_tile_rows(H, G, D, Dv, dtype)}:
            plan = ops.prefill_plan(cq, sum(qlens), max(qlens), rows)
            for use, ref in ((None, want), (gc[:, 3:3 + H], gated)):
                got = ops.sigmoid_attention(qc, kc, vc, cq, cu(klens).cuda(), max(qlens), scale, bias.cuda(), chunk, use, plan=plan)
                ops.check_status()
                close(got, ref, TOL[dtype])


@pytest.mark.parametrize("D", [128, 64, 40])
def test_sigmoid_weights_at_the_ends_of_their_range(D):
    """Scores far below zero give weights of no more than their own size, scores far above give ones; nothing overflows."""
    from llm_from_scratch_b200 import ops
    n = 150
    q, k = torch.zeros(n, 1, D), torch.zeros(n, 1, D)
    q[:, 0, 0], k[:, 0, 0] = 1.0, torch.linspace(-3000, 300, n)
    v = torch.ones(n, 1, D)
    args = [x.bfloat16().cuda() for x in (q, k, v)]
    c = cu([n]).cuda()
    got = ops.sigmoid_attention(*args, c, c, n, 1.0, torch.tensor([0.5]).cuda(), 0)
    want = orc.sigmoid_attention(*(x.cpu().double() for x in args), 1.0, torch.tensor([0.5]).double())
    assert torch.isfinite(got).all() and (got.cpu().double() - want).abs().max() < 0.05 and got[:100].abs().max() < 1e-15
    low = ops.sigmoid_attention(*args[:2], args[2], c, c, n, 0.0, torch.tensor([-9.0]).cuda(), 0)       # all weights e^-9
    close(low[:, 0, 0], torch.arange(1, n + 1) / (1 + torch.tensor(9.0).exp()), 1e-2)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("bs", [16, 64, 24])
@pytest.mark.parametrize("H,G,D,Dv", [(8, 2, 128, 128), (16, 1, 64, 64), (6, 6, 32, 32), (20, 2, 128, 128), (4, 2, 24, 24), (3, 1, 7, 11),
                                      (4, 1, 200, 200)])
def test_sigmoid_decode(H, G, D, Dv, bs, dtype):
    """Contexts at block and chunk borders, cut over many CTAs; single sequences and batches beyond the in-launch merge."""
    from llm_from_scratch_b200 import ops
    g, scale = gen(D + bs), 1.5 * D ** -0.5
    lens = [1, 16, 0, 65, 1500, 333, 64, 100, 101, 200, 201]
    bias = torch.linspace(-2.0, 1.0, H)
    bt, nb = tables(lens, bs)
    k = torch.randn(nb * bs, G, D, generator=g)
    for chunk in (0, 1, 15, 16, 17, 64, 100, 1000):
        v = torch.randn(nb * bs, G, Dv, generator=g)
        for i, n in enumerate(lens):
            if n:
                at = slots_of(bt, i, n, bs)
                v[at] = edges(v[at], chunk)
        kc, vc = (x.to(dtype).view(nb, bs, G, -1).cuda() for x in (k, v))
        for which in ([4], [0, 5], list(range(11)), list(range(11)) * 4):
            q = torch.randn(len(which), H, D, generator=g).to(dtype)
            gate = (2 * torch.randn(len(which), H + 3, generator=g)).to(dtype)
            got = ops.sigmoid_decode(q.cuda(), kc, vc, bt[which].cuda(), torch.tensor([lens[i] for i in which]).cuda(), scale, bias.cuda(),
                                     chunk, gate.cuda()[:, 1:1 + H])
            ops.check_status()
            for r, i in enumerate(which[:11]):
                n = lens[i]
                if n == 0:
                    assert not got[r].any()
                    continue
                at = slots_of(bt, i, n, bs)
                want = orc.sigmoid_attention(q[r:r + 1].double(), k[at].to(dtype).double(), v[at].to(dtype).double(), scale, bias.double(),
                                             chunk, n - 1)[0]
                close(got[r], want * torch.sigmoid(gate[r, 1:1 + H].double())[:, None], TOL[dtype])


# -------------------------------------------------------------------------------------------- experts
@pytest.mark.parametrize("T", [1, 7, 128, 129, 2500])
@pytest.mark.parametrize("E,top", [(12, 3), (16, 2), (64, 8), (300, 6), (5, 5), (6, 1), (1, 1), (40, 32)])
def test_softmax_route(E, top, T):
    from llm_from_scratch_b200 import ops
    g = gen(E + T)
    z, bias = 3 * torch.randn(T, E, generator=g) - 20.0, torch.randn(E, generator=g)
    tok, w, offs, slot = (t.cpu() for t in ops.moe_softmax_route(z.cuda(), bias.cuda(), top))
    expert_of = torch.bucketize(slot.long(), offs.long(), right=True)                                # [T, top], in order of choice
    for t, (chosen, wts, _) in enumerate(orc.route((z + bias)[:min(T, 150)], torch.eye(E), torch.zeros(E), top)):
        assert expert_of[t].tolist() == chosen
        assert torch.allclose(w[t].double(), wts.double(), rtol=1e-5)
    assert int(offs[-1]) == T * top and sorted(slot.reshape(-1).tolist()) == list(range(T * top))
    assert torch.equal(tok[slot.long()], torch.arange(T).int()[:, None].expand(T, top))


def test_equal_logits_go_to_the_lower_expert():
    from llm_from_scratch_b200 import ops
    tok, w, offs, slot = (t.cpu() for t in ops.moe_softmax_route(torch.zeros(2, 6).cuda(), torch.zeros(6).cuda(), 3))
    assert torch.bucketize(slot.long(), offs.long(), right=True).tolist() == [[0, 1, 2]] * 2 and torch.allclose(w, torch.tensor(1 / 3))


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("counts,k,n", [([5, 0, 17, 1], 120, 40), ([130, 0, 3], 64, 200), ([400, 300], 256, 384), ([9, 70, 0, 0, 2], 33, 21),
                                        ([0, 0, 1], 8, 8), ([90, 1, 200], 100, 36)])
def test_grouped_linear_with_squared_relu(counts, k, n, dtype):
    from llm_from_scratch_b200 import ops
    g, E, R = gen(k + n), len(counts), sum(counts)
    x = torch.randn(R, k, generator=g).to(dtype)
    w = (2 * torch.randn(E, n, k, generator=g) * k ** -0.5).to(dtype)
    offs = torch.tensor(counts).cumsum(0).int()
    want = torch.cat([(part @ w[e].double().T).clamp(min=0) ** 2 for e, part in enumerate(x.double().split(counts))])
    got = ops.moe_grouped_linear(x.cuda(), w.cuda(), offs.cuda(), squared_relu=True)
    ops.check_status()
    close(got, want, TOL[dtype])
