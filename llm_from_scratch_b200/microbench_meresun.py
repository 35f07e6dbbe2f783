"""Timed runs of the Meresun family: its kernels on layer sizes of real models beside the like kernels of the other families, and
prefill / decode throughput of the whole model beside the MLA + MoE decoder of equal width, heads, ranks, experts and depth
(``bench.py --workload meresun`` and ``meresun_kernels``).  Weights are random; inputs of the kernel runs exceed the L2 or rotate
over buffers that do."""
from __future__ import annotations

import itertools

import numpy as np
import torch

from . import ops
from .microbench_nabalix import VOCAB, _time, _visible_pairs, engine_rates

# width, heads of 128 + 64 rotary channels, query and key / value rank, feed-forward of an expert and of the MLA model's dense
# layers (the PolyNorm feed-forward is half as wide again: equal parameters), experts, experts per token, groups, kept groups
SIZES = {
    "d1024": dict(d=1024, H=8, rq=512, r=512, ff=1408, E=16, K=2, groups=4, keep=2),
    "d2048": dict(d=2048, H=16, rq=1024, r=512, ff=1408, E=32, K=4, groups=4, keep=2),
    "d4096": dict(d=4096, H=32, rq=1536, r=512, ff=2048, E=32, K=4, groups=8, keep=4),
}
DIM, ROT, VDIM, WINDOW, SIDE = 128, 64, 128, 512, 256
YARN = dict(factor=8.0, original=4096, fast=32.0, slow=1.0)


def meresun_config(z: dict, layers: int, window: int = WINDOW) -> dict:
    mixer = dict(heads=z["H"], dim=DIM, rot_dim=ROT, vdim=VDIM, q_rank=z["rq"], kv_rank=z["r"], scale=(DIM + ROT) ** -0.5,
                 rot=dict(dims=ROT, base=5e5, scaling=YARN), mask=dict(size=window) if window else None)
    dense = {"kind": "dense", "ff": z["ff"] * 3 // 2}
    moe = {"kind": "moe", "expert": dict(ff=z["ff"], limit=7.0),
           "router": dict(experts=z["E"], top=z["K"], groups=dict(count=z["groups"], keep=z["keep"]))}
    return {"architecture": "Meresun", "vocab": VOCAB, "width": z["d"], "norm": {"eps": 1e-5, "groups": 2},
            "embedding": {"scale": 1.0}, "token_side": {"dim": SIDE},
            "layers": [{"type": "latent_attention", "mixer": mixer, "mlp": moe if i % 2 else dense} for i in range(layers)]}


def mla_config(z: dict, layers: int) -> dict:
    return dict(vocab_size=VOCAB, context_length=8192, d_model=z["d"], num_layers=layers, num_heads=z["H"], d_ff=z["ff"],
                attention_type="MLA", rope_dim=ROT, q_lora_rank=z["rq"], kv_lora_rank=z["r"], use_moe=True,
                moe_layers=list(range(1, layers, 2)), n_routed_experts=z["E"], num_experts_per_tok=z["K"], n_shared_experts=0)


def kernels(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), hbm_gbs: float = 6547.0,
            tflops: float = 1654.0) -> dict:
    """Every kernel of the family alone: ragged prompts (8 of 1024 tokens), decode at 64 and 256 sequences with full windows;
    each followed by the like kernel of another family on the same shape (windows: the same number of visible keys)."""
    dev, dt, bs, n = torch.device("cuda"), torch.bfloat16, 64, 8
    out = {}
    for name in sizes:
        z = SIZES[name]
        d, H, rq, r, F, E, K = z["d"], z["H"], z["rq"], z["r"], z["ff"], z["E"], z["K"]
        gen = torch.Generator(device=dev).manual_seed(1)
        rnd = lambda *s, dtype=dt: torch.randn(*s, generator=gen, device=dev, dtype=dtype)
        ones = lambda k: torch.ones(k, device=dev)
        res = {}

        def mem(key, fn, nbytes, reps=steps):
            ms = _time(fn, reps, warmup)
            res[key] = dict(us=ms * 1e3, gbs=nbytes / ms / 1e6, frac=nbytes / ms / 1e6 / hbm_gbs)

        def tensor(key, fn, flops):
            ms = _time(fn, steps, warmup)
            res[key] = dict(us=ms * 1e3, tflops=flops / ms / 1e9, frac=flops / ms / 1e9 / tflops)

        # ---- prompts: attention over packed keys, also at the end of longer contexts
        lens = [1024] * n
        T = sum(lens)
        cu = torch.tensor(np.concatenate([[0], np.cumsum(lens)]), dtype=torch.int32, device=dev)
        slots, pos = torch.arange(T, device=dev), torch.arange(T, device=dev) % 1024
        sink = torch.zeros(H, device=dev)
        q, kh, kt, v = rnd(T, H, DIM + ROT), rnd(T, H, DIM), rnd(T, ROT), rnd(T, H, VDIM)
        plan = ops.prefill_plan(cu, T, 1024, ops.prefill_window_tile_rows(H, H, DIM + ROT, ROT, VDIM, dt))
        flop = H * 2 * (DIM + ROT + VDIM)
        for w in (0, WINDOW, 128):
            tensor(f"prefill_attention_w{w}", lambda: ops.prefill_varlen_window(q, kh, kt, v, cu, cu, 1024, 0.05, w, sink, plan=plan),
                   _visible_pairs(lens, w or 1 << 30) * flop)
        tensor("prefill_attention.mla", lambda: ops.prefill_varlen_shared_tail(q, kh, kt, v, cu, cu, 1024, 0.05, plan=plan),
               _visible_pairs(lens, 1 << 30) * flop)
        del kh, v
        # a head size of its own, on the mma.sync kernel, beside the same kernel at its compiled size
        qs, ks, ts, vs = rnd(T, H, 96), rnd(T, H, 64), rnd(T, 32), rnd(T, H, 96)
        plan64 = ops.prefill_plan(cu, T, 1024, 64)
        tensor("prefill_attention_96", lambda: ops.prefill_varlen_window(qs, ks, ts, vs, cu, cu, 1024, 0.05, 0, sink, plan=plan64),
               _visible_pairs(lens, 1 << 30) * H * 2 * 192)
        k64, v64 = rnd(T, H, 64), rnd(T, H, 64)
        tensor("prefill_attention_96.gqa64", lambda: ops.prefill_varlen(qs[..., :64].contiguous(), k64, v64, cu, cu, 1024, 1024, 0.05, plan=plan64),
               _visible_pairs(lens, 1 << 30) * H * 2 * 128)
        del qs, ks, ts, vs, k64, v64
        # ---- prologue
        rot = ops.Rotation(5e5, ROT, dev, ops.YarnScaling(**{k: float(x) for k, x in YARN.items()}))
        proj, pool = rnd(T, rq + r + ROT + 2 * d), rnd(T // bs, bs, r + ROT)
        dq, dkv = proj[:, :rq], proj[:, rq:rq + r + ROT]
        mem("latent_prologue", lambda: ops.latent_prologue(dq, ones(rq), dkv, ones(r), 1e-5, rot, pos, pool, slots),
            T * (2 * rq + 3 * (r + ROT)) * 2)
        mem("rotate_heads", lambda: ops.rotate_heads(q, ROT, rot, pos), T * H * ROT * 4)
        table = torch.zeros(1024, DIM, device=dev)
        qf, kvp, cq = rnd(T, H * (DIM + ROT)), rnd(T, r + ROT), rnd(T, rq)
        mem("prologue.mla", lambda: ops.mla_prologue(qf, kvp, ones(r), table, pos, H, DIM, ROT, r, pool, slots),
            T * (2 * H * (DIM + ROT) + 3 * (r + ROT)) * 2)
        mem("query_norm.mla", lambda: ops.add_rmsnorm(cq, ones(rq), 1e-5), T * rq * 4)
        del q, qf, kvp, cq
        bt = torch.randperm(T // bs, generator=gen, device=dev).int().view(n, -1)
        ends = torch.arange(n + 1, dtype=torch.int32, device=dev) * 700
        mem("gather_last_rows", lambda: ops.gather_rows(pool, bt, ends, 700, 700 * n, cu), n * 700 * (r + ROT) * 4)
        # ---- residual, gates, activations, token input
        x, y, y2, nw = torch.zeros(T, d, device=dev), rnd(T, d), rnd(T, d), ones(d)
        g1, g2 = proj[:, -2 * d:-d], proj[:, -d:]
        mem("residual_group_norm", lambda: ops.residual_group_norm(x, nw, 2, 1e-5, dt, y=y, y_norm_w=nw), T * d * 12)
        mem("residual.mla", lambda: ops.add_rmsnorm(y, nw, 1e-5, y2), T * d * 8)
        mem("gated_residual", lambda: ops.gated_residual(x, y, g1, y2, g2), T * d * 18)
        rows, wts = rnd(T * K, d), torch.rand(T, K, device=dev)
        slot = torch.randperm(T * K, generator=gen, device=dev).int().view(T, K)
        mem("gated_residual_experts", lambda: ops.gated_residual(x, y, g1, rows, g2, wts, slot), T * d * (16 + 2 * K))
        rexp, rw = torch.zeros(T * K, dtype=torch.int32, device=dev), rnd(T * K)
        mem("combine.mla", lambda: ops.moe_combine(rows, None, rexp, rw, slot), T * d * (2 + 2 * K))
        del rows, y2
        up, gu, coef = rnd(T, F * 3 // 2), rnd(T, 2 * F), torch.tensor([0.6, 0.4, 0.2, 0.1], device=dev)
        mem("poly_norm", lambda: ops.poly_norm(up, coef, 1e-5), T * F * 6)
        mem("poly_norm.mla", lambda: ops.swiglu(gu), T * F * 6)
        del up, gu
        u, side, ids = rnd(T, SIDE), rnd(VOCAB, 4 * SIDE), torch.randint(0, VOCAB, (T,), device=dev)
        mem("gelu_table", lambda: ops.gelu_table(u, side, SIDE, ids), T * SIDE * 6)
        # ---- experts
        w_in, w_down = rnd(E, 2 * F, d), rnd(E, d, F)
        corr = torch.zeros(E, device=dev)
        for tokens in (64, 256, 2048, 8192):
            logits = rnd(tokens, E, dtype=torch.float32)
            lb = logits.to(dt)
            res[f"route_{tokens}"] = dict(us=_time(lambda: ops.moe_group_route(logits, corr, K, z["groups"], z["keep"]), steps, warmup) * 1e3)
            res[f"route.mla_{tokens}"] = dict(us=_time(lambda: ops.moe_route(lb, corr, K), steps, warmup) * 1e3)
            if tokens * K > 256 * E:
                continue
            tok, _, offs, _ = ops.moe_group_route(logits, corr, K)
            xs = rnd(tokens, d).index_select(0, tok)
            act = rnd(tokens * K, F)
            hit = int((offs.diff(prepend=offs.new_zeros(1)) > 0).sum())
            flops, nbytes = tokens * K * d * F * 2, hit * d * F * 2
            for key, fn, parts in (("experts_up", lambda: ops.moe_grouped_linear(xs, w_in, offs, glu=(7.0, 1.702)), 2),
                                   ("experts_up.mla", lambda: ops.moe_grouped_gemm(xs, w_in, offs, swiglu=True), 2),
                                   ("experts_down", lambda: ops.moe_grouped_linear(act, w_down, offs), 1),
                                   ("experts_down.mla", lambda: ops.moe_grouped_gemm(act, w_down, offs), 1)):
                if tokens <= 256:
                    mem(f"{key}_{tokens}", fn, nbytes * parts)
                else:
                    tensor(f"{key}_{tokens}", fn, flops * parts)
        del w_in, w_down
        # ---- decode: contexts twice the window; the like kernel has contexts of one window
        for B in (64, 256):
            it = itertools.count()
            nbk = 2 * WINDOW // bs
            sets = int(300e6 / (B * WINDOW * (r + ROT) * 2)) + 1               # rotate pools larger than the L2
            pools = [rnd(B * nbk, bs, r + ROT) for _ in range(sets)]
            bts = torch.randperm(B * nbk, generator=gen, device=dev).int().view(B, nbk)
            long, short = (torch.full((B,), c, dtype=torch.int64, device=dev) for c in (2 * WINDOW, WINDOW))
            qa, qr = rnd(B, H, r), rnd(B, H, ROT)
            nbytes = B * WINDOW * (r + ROT) * 2
            mem(f"decode_attention_{B}", lambda: ops.mla_decode(qa, qr, pools[next(it) % sets], bts, long, 0.05, window=WINDOW, sink=sink),
                nbytes, 3 * steps)
            mem(f"decode_attention.mla_{B}", lambda: ops.mla_decode(qa, qr, pools[next(it) % sets], bts, short, 0.05), nbytes, 3 * steps)
            small = [p.view(-1, 16, r + ROT) for p in pools]
            bt16 = (bts[:, :, None] * 4 + torch.arange(4, device=dev)).reshape(B, -1).int().contiguous()
            mem(f"decode_attention.mla16_{B}", lambda: ops.mla_decode(qa, qr, small[next(it) % sets], bt16, short, 0.05), nbytes, 3 * steps)
            del pools, small
        ops.check_status()
        torch.cuda.empty_cache()
        out[name] = res
    return dict(workload="Meresun kernels alone, bf16; '.family' rows are the like kernels of other families",
                sizes={n: SIZES[n] for n in sizes}, kernels=out)


def throughput(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), layers: int = 4, batch: int = 64,
               prompt: int = 1024) -> dict:
    """Prefill and decode throughput through the engine: ``layers`` layers of every size (dense and mixture of experts in
    turns), prompts of ``prompt`` tokens eight to a step, then ``batch`` sequences decoding from captured graphs; beside the
    MLA + MoE decoder of the same width, heads, ranks, experts and depth (full attention, SwiGLU, no gates or token input)."""
    from .model import resolve_config
    from .model.meresun import init_weights
    out = {}
    for name in sizes:
        cfg = meresun_config(SIZES[name], layers)
        weights = init_weights(resolve_config(cfg), 0, torch.bfloat16)
        a = engine_rates(cfg, weights, 64, steps, warmup, batch, prompt)
        b = engine_rates(mla_config(SIZES[name], layers), None, 16, steps, warmup, batch, prompt)
        out[f"{name}.meresun"], out[f"{name}.mla"] = a, b
        out[f"{name}.ratio"] = dict(prefill=a["prefill_tokens_per_s"] / b["prefill_tokens_per_s"],
                                    decode=a["decode_tokens_per_s"] / b["decode_tokens_per_s"])
    return dict(workload=f"engine throughput, {layers} layers, window {WINDOW}, prefill steps of 8 prompts x {prompt} tokens, "
                         f"decode of {batch} sequences with contexts from {prompt}, bf16, random weights", results=out)
