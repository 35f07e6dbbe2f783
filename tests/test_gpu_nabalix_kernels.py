"""The CUDA mechanisms of the Nabalix family against the plain CPU restatement, each alone."""
import numpy as np
import pytest
import torch

from oracle import nabalix as orc

pytestmark = pytest.mark.gpu


def gen(seed):
    return torch.Generator().manual_seed(seed)


def rel(a, b):
    return ((a.double().cpu() - b).abs().max() / b.abs().max().clamp(min=1e-6)).item()


# ------------------------------------------------------------------------------------------ streams
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-6), (torch.bfloat16, 6e-3)])
@pytest.mark.parametrize("S,d", [(1, 64), (2, 112), (3, 99), (4, 2048), (6, 40)])
def test_stream_update(S, d, dtype, tol):
    from llm_from_scratch_b200 import ops
    T, eps = 7, 1e-5
    g = gen(S)
    emb = torch.randn(11, d, generator=g).to(dtype)
    ids = torch.randint(0, 11, (T,), generator=g)
    r = lambda *s: torch.randn(*s, generator=g)
    nw, ls, w0, w1, win, wout, mix = r(d) * 0.3, r(d), r(d), r(d), r(S), r(S), r(S, S)
    y0, y1 = r(T, d).to(dtype), (r(T, d) * 5).to(dtype)
    c = lambda t: t.cuda()
    X = torch.zeros(T, S, d).cuda()
    h = ops.stream_update(X, c(nw), eps, dtype, tokens=c(ids), embed=c(emb), in_w=c(win))
    want = emb.double()[ids][None].repeat(S, 1, 1)
    assert torch.equal(X.cpu().double(), want.transpose(0, 1))
    assert rel(h, orc.norm_one_plus(orc.streams_read(want, win.double()), nw.double(), eps)) < tol
    for second in (False, True):      # one result, then the join of two; the last call reads the plain sum
        y = orc.parallel_join(y0.double(), y1.double(), w0.double(), w1.double(), eps) if second else y0.double()
        want = orc.streams_write(want, y * ls.double(), mix.double(), wout.double())
        h = ops.stream_update(X, c(nw), eps, dtype, y=c(y0), y1=c(y1) if second else None,
                              join_w=(c(w0), c(w1)) if second else None, join_eps=eps, layer_scale=c(ls), mix=c(mix),
                              out_w=c(wout), in_w=None if second else c(win))
        u = want.sum(0) if second else orc.streams_read(want, win.double())
        assert rel(X.transpose(0, 1), want) < 3e-6
        assert rel(h, orc.norm_one_plus(u, nw.double(), eps)) < tol
    ops.check_status()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 1e-6), (torch.bfloat16, 5e-3)])
@pytest.mark.parametrize("F", [8, 80, 77])
def test_clamped_glu(F, dtype, tol):
    from llm_from_scratch_b200 import ops
    h = (torch.randn(9, 2 * F, generator=gen(F)) * 3).to(dtype)
    want = orc.clamped_glu(h[:, :F].double(), h[:, F:].double(), 1.3)
    assert rel(ops.clamped_glu(h.cuda(), 1.3, 1.702), want) < tol


# ---------------------------------------------------------------------------------------- attention
class Pool:
    """A paged pool that holds the contexts of several sequences in shuffled blocks, with stale rows elsewhere."""

    def __init__(self, lens, G, dk, dv, bs, dtype, seed):
        g = gen(seed)
        self.k = [torch.randn(n, G, dk, generator=g).to(dtype) for n in lens]
        self.v = [torch.randn(n, G, dv, generator=g).to(dtype) for n in lens]
        blocks = [(n + bs - 1) // bs for n in lens]
        order = torch.randperm(sum(blocks) + 3, generator=g)
        self.kc = torch.full((sum(blocks) + 3, bs, G, dk), 50.0, dtype=dtype)
        self.vc = torch.full((sum(blocks) + 3, bs, G, dv), 50.0, dtype=dtype)
        self.bt = torch.full((len(lens), max(blocks + [1]) + 1), -1, dtype=torch.int32)
        at = 0
        for s, nb in enumerate(blocks):
            ids = order[at:at + nb]
            at += nb
            self.bt[s, :nb] = ids.int()
            for j in range(lens[s]):
                self.kc[ids[j // bs], j % bs] = self.k[s][j]
                self.vc[ids[j // bs], j % bs] = self.v[s][j]

    def cuda(self):
        return self.kc.cuda(), self.vc.cuda(), self.bt.cuda()


def head_constants(H, seed):
    """r1, r2, talk; for some head counts talk is not exact in bf16 (another form of the mix serves it)."""
    g = gen(seed + 77)
    talk = torch.eye(H) + 0.3 * torch.randn(H, H, generator=g)
    return (torch.rand(H, generator=g).bfloat16().float(), torch.rand(H, generator=g).bfloat16().float(),
            talk if H in (12, 28) else talk.bfloat16().float())


SHAPES = [  # H, G, dk, dv, window, block size
    (4, 2, 32, 48, 40, 16), (6, 2, 64, 112, 50, 64), (1, 1, 16, 16, 1, 16), (8, 8, 48, 32, 7, 16),
    (16, 4, 64, 64, 100, 16), (12, 2, 128, 128, 64, 32), (24, 4, 64, 32, 33, 16), (32, 2, 32, 64, 70, 16),
    (5, 1, 80, 96, 0, 16), (3, 3, 20, 24, 10, 16), (16, 16, 32, 32, 0, 64), (9, 3, 256, 256, 90, 16), (16, 1, 64, 64, 48, 16),
    (28, 4, 32, 32, 60, 16), (16, 4, 128, 128, 130, 16), (32, 8, 128, 128, 130, 64)]


@pytest.mark.parametrize("general", [False, True])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,G,dk,dv,window,bs", SHAPES)
def test_talking_attention(H, G, dk, dv, window, bs, dtype, general):
    """Ragged portions behind contexts of unequal lengths (one a single token), and the same last tokens through
    the decode form; one score stands out just inside the window's edge, and one just outside it."""
    from llm_from_scratch_b200 import ops
    if general and dtype == torch.float32:
        pytest.skip("fp32 always runs the general kernel")
    klens, qlens = [150, 37, 1, 201, 64], [70, 37, 1, 1, 2]
    scale, cap = dk ** -0.5, 15.0
    r1, r2, talk = head_constants(H, H)
    pool = Pool(klens, G, dk, dv, bs, dtype, seed=H + dk)
    g = gen(5)
    q = [torch.randn(n, H, dk, generator=g).to(dtype) for n in qlens]
    if window > 1:            # the last query of every sequence matches the keys at both sides of the window's edge
        for s, n in enumerate(klens):
            q[s][-1] = torch.ones(H, dk) * 2
            for back in (window - 1, window):
                if 0 <= n - 1 - back:
                    j = n - 1 - back
                    pool.k[s][j] = 1.0
                    pool.v[s][j] = 3.0 if back == window else -3.0
                    b = pool.bt[s, j // bs]
                    pool.kc[b, j % bs], pool.vc[b, j % bs] = pool.k[s][j], pool.v[s][j]
    gate = torch.randn(sum(qlens), H * dv, generator=g).to(dtype)
    d = lambda t: t.double()
    want = torch.cat([orc.attention(d(q[s]), d(pool.k[s]), d(pool.v[s]), scale, cap, d(r1), d(r2), d(talk), window,
                                    first=klens[s] - qlens[s]) for s in range(5)])
    want = want * torch.sigmoid(d(gate)).view(-1, H, dv)
    kc, vc, bt = pool.cuda()
    c = ops.TalkingHeads(scale, cap, r1, r2, talk, window, "cuda")
    Q = torch.cat(q).reshape(-1, H * dk).cuda()
    cu = lambda x: torch.tensor(np.concatenate([[0], np.cumsum(x)]), dtype=torch.int32).cuda()
    pad = lambda t: torch.cat([t, torch.zeros(5, t.shape[1], dtype=t.dtype, device=t.device)])   # padding rows
    got = ops.talking_attention(pad(Q), pad(gate.cuda()), kc, vc, bt, c, cu_seqlens_q=cu(qlens), cu_seqlens_k=cu(klens),
                                max_seqlen_q=70, general=general)[:sum(qlens)]
    ops.check_status()
    tol = 1e-5 if dtype == torch.float32 else 1.2e-2
    assert rel(got, want) < tol
    plan = ops.prefill_plan(cu(qlens), sum(qlens) + 5, 70, ops.TALKING_TILE_ROWS)
    again = ops.talking_attention(pad(Q), pad(gate.cuda()), kc, vc, bt, c, cu_seqlens_q=cu(qlens), cu_seqlens_k=cu(klens),
                                  max_seqlen_q=70, plan=plan, general=general)[:sum(qlens)]
    assert torch.equal(again, got)
    # decode form: the last row of every sequence, plus padding rows of a captured batch
    last = torch.tensor(np.cumsum(qlens) - 1)
    lens = torch.tensor(klens + [0, 0]).cuda()
    bt2 = torch.cat([bt, bt[:2]])
    got = ops.talking_attention(torch.cat([Q[last.cuda()], Q[:2]]), torch.cat([gate[last], gate[:2]]).cuda(), kc, vc, bt2,
                                c, context_lens=lens, general=general)[:5]
    ops.check_status()
    assert rel(got, want[last]) < tol


def test_talking_attention_without_gate_and_cap_and_with_scores_that_outgrow_the_first_tile():
    """Later keys beat the first tile's maximum by far more than the lazy maximum tolerates, in both directions."""
    from llm_from_scratch_b200 import ops
    H, G, dk, dv, n = 8, 2, 32, 32, 200
    for sign in (1, -1):
        pool = Pool([n], G, dk, dv, 16, torch.bfloat16, seed=3)
        ramp = torch.linspace(-6, 6, n)[:, None, None] * sign
        pool.k[0] = (ramp * torch.ones(1, G, dk)).bfloat16()
        for j in range(n):
            pool.kc[pool.bt[0, j // 16], j % 16] = pool.k[0][j]
        q = torch.ones(40, H, dk).bfloat16()
        r1, r2, talk = head_constants(H, 1)
        d = lambda t: t.double()
        s = torch.einsum("ihd,jhd->hij", d(q), d(pool.k[0])[:, torch.arange(H) // 4]) * 0.5
        dist = torch.arange(n - 40, n)[:, None] - torch.arange(n)[None]
        s = torch.einsum("hg,gij->hij", d(talk), s - orc.distance_bias(d(r1), d(r2), dist.clamp(min=0)))
        p = torch.softmax(s.masked_fill((dist < 0)[None], -torch.inf), -1)
        want = torch.einsum("hij,jhd->ihd", p, d(pool.v[0])[:, torch.arange(H) // 4])
        kc, vc, bt = pool.cuda()
        c = ops.TalkingHeads(0.5, 0.0, r1, r2, talk, 0, "cuda")
        cu = lambda x: torch.tensor([0, x], dtype=torch.int32).cuda()
        Q = q.reshape(40, -1).cuda()
        got = ops.talking_attention(Q, None, kc, vc, bt, c, cu_seqlens_q=cu(40), cu_seqlens_k=cu(n), max_seqlen_q=40)
        assert rel(got, want) < 1.2e-2
        got = ops.talking_attention(Q[-1:], None, kc, vc, bt, c, context_lens=torch.tensor([n]).cuda())
        assert rel(got, want[-1:]) < 1.2e-2


# --------------------------------------------------------------------------------------- recurrence
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 2e-5), (torch.bfloat16, 1e-2)])
@pytest.mark.parametrize("H,dk,dv", [(3, 16, 32), (5, 48, 40), (1, 1, 1), (2, 80, 64), (4, 128, 128), (2, 200, 72), (1, 40, 264),
                                     (2, 33, 30)])
def test_gated_recurrence_in_portions_and_steps(H, dk, dv, dtype, tol):
    """Unequal sequences in one batch, cut into portions (long ones span several scan segments, one is a single
    token), then decoded token by token; slots start with garbage, move by a permutation, and gates reach both ends."""
    from llm_from_scratch_b200 import ops
    eps, n = 1e-5, 4
    g = gen(dk)
    lens = [300, 41, 7, 2]
    w = H * dk
    r = lambda *s: torch.randn(*s, generator=g)
    fb, lower, nw = r(w) * 3, torch.rand(w, generator=g), r(dv)
    lower[:: 5] = 0
    proj = [r(m, 2 * w + H * dv).to(dtype) * 2 for m in lens]
    d = lambda t: t.double()
    want = []
    for p in proj:
        q = orc.silu(d(p[:, :w])).view(-1, H, dk)
        f = orc.forget_gate(d(p[:, w:2 * w]), d(fb), d(lower)).view(-1, H, dk)
        o, S = orc.gated_recurrence(q, f, d(p[:, 2 * w:]).view(-1, H, dv))
        want.append((orc.norm_plain(o, d(nw), eps).reshape(len(p), -1), S))
    state = torch.full((6, H, dk, dv), 7.0).cuda()
    slots = torch.tensor([4, 0, 5, 2]).cuda()
    args = (fb.cuda(), lower.cuda(), nw.cuda(), eps, state, slots)
    cut = [[0, 170, 171, 290], [0, 30, 32, 35], [0, 1, 3, 6], [0, 1, 1, 1]]
    cu = lambda x: torch.tensor(np.concatenate([[0], np.cumsum(x)]), dtype=torch.int32).cuda()
    got = [[] for _ in range(n)]
    for i in range(3):
        ql = [cut[s][i + 1] - cut[s][i] for s in range(n)]
        x = torch.cat([proj[s][cut[s][i]:cut[s][i + 1]] for s in range(n)]).cuda()
        y = ops.gated_recurrence(x[:, :w], x[:, w:2 * w], x[:, 2 * w:], *args, cu_seqlens_q=cu(ql),
                                 cu_seqlens_k=cu([cut[s][i + 1] for s in range(n)]), max_seqlen_q=max(ql))
        for s, part in enumerate(y.split(ql)):
            got[s].append(part)
    for k in range(10):
        at = [cut[s][3] + k for s in range(n)]
        x = torch.stack([proj[s][min(at[s], lens[s] - 1)] for s in range(n)]).cuda()
        live = torch.tensor([a + 1 if a < lens[s] else 0 for s, a in enumerate(at)]).cuda()
        y = ops.gated_recurrence(x[:, :w], x[:, w:2 * w], x[:, 2 * w:], *args, context_lens=live)
        for s in range(n):
            if at[s] < lens[s]:
                got[s].append(y[s:s + 1])
    ops.check_status()
    for s in range(n):
        assert rel(torch.cat(got[s])[:lens[s]], want[s][0]) < tol
        assert rel(state[slots[s]], want[s][1]) < (2e-5 if dtype == torch.float32 else 2e-5)
    assert (state[[1, 3]] == 7.0).all()


def test_store_kv_rows_of_unequal_widths():
    from llm_from_scratch_b200 import ops
    for wk, wv, dtype in ((64, 96, torch.bfloat16), (21, 10, torch.bfloat16), (12, 20, torch.float32), (3, 5, torch.float32)):
        x = torch.randn(5, wk + wv + 8, generator=gen(wk)).to(dtype).cuda()
        kc, vc = torch.zeros(2, 4, 1, wk, dtype=dtype).cuda(), torch.zeros(2, 4, 1, wv, dtype=dtype).cuda()
        slots = torch.tensor([3, -1, 7, 0, 4]).cuda()
        ops.store_kv_rows(x[:, :wk], x[:, wk:wk + wv], kc, vc, slots)
        for t, s in enumerate(slots.tolist()):
            if s >= 0:
                assert torch.equal(kc.view(8, wk)[s], x[t, :wk]) and torch.equal(vc.view(8, wv)[s], x[t, wk:wk + wv])
        assert (kc.view(8, wk)[[1, 2, 5, 6]] == 0).all()
        ops.check_status()
