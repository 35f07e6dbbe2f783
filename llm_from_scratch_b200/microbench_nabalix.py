"""Timed runs of the Nabalix family: its kernels on layer sizes of real models, and prefill / decode throughput of
the whole model beside the GQA decoder of equal width, heads, feed-forward and depth (``bench.py --workload
nabalix`` and ``nabalix_kernels``).  Weights are random; inputs of the kernel runs exceed the L2 or rotate over
buffers that do."""
from __future__ import annotations

import itertools
import time

import numpy as np
import torch

from . import ops


def _time(fn, steps: int, warmup: int) -> float:
    """Milliseconds per call of ``fn``, ``steps`` calls replayed from one CUDA graph (no host work in between)."""
    for _ in range(max(warmup, 1)):
        fn()
    torch.cuda.synchronize()
    graph = torch.cuda.CUDAGraph()
    with torch.cuda.graph(graph):
        for _ in range(steps):
            fn()
    graph.replay()
    torch.cuda.synchronize()
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    e0.record()
    graph.replay()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / steps

# (width, heads, kv heads, head size, recurrence heads x size, d_ff, window)
SIZES = {
    "d1024": dict(d=1024, H=16, G=4, dim=64, rec=(8, 64, 64), ff=2816, window=1024),
    "d2048": dict(d=2048, H=16, G=4, dim=128, rec=(16, 128, 128), ff=5632, window=1024),
    "d4096": dict(d=4096, H=32, G=8, dim=128, rec=(16, 128, 128), ff=11264, window=2048),
}
VOCAB, STREAMS = 32000, 4


def nabalix_config(size: dict, layers: int) -> dict:
    layer = {"type": "parallel",
             "mixer": {"left": {"heads": size["H"], "kv_heads": size["G"], "dim": size["dim"], "vdim": size["dim"],
                                "scale": size["dim"] ** -0.5, "softcap": 30.0, "mask": {"size": size["window"]}},
                       "right": dict(zip(("heads", "dim", "vdim"), size["rec"]))},
             "mlp": {"kind": "dense", "ff": size["ff"], "limit": 7.0}}
    return {"architecture": "Nabalix", "vocab": VOCAB, "width": size["d"], "streams": STREAMS, "norm": {"eps": 1e-5},
            "layers": [layer] * layers}


def gqa_config(size: dict, layers: int) -> dict:
    return dict(vocab_size=VOCAB, context_length=8192, d_model=size["d"], num_layers=layers, num_heads=size["H"],
                num_kv_heads=size["G"], d_ff=size["ff"], attention_type="GQA", use_moe=False)


def _visible_pairs(lens, window: int) -> int:
    return int(sum(n * (n + 1) // 2 - max(n - window, 0) * (max(n - window, 0) + 1) // 2 for n in map(int, lens)))


def talking_roofline_us(pairs: int, H: int, dk: int, dv: int, tflops: float, sms: int = 148, mhz: float = 1965.0) -> dict:
    """Lower bounds of the prefill attention in us: tensor pipe (QK, PV), fp32 pipe (H x H mix and at least eight
    operations per score) and special-function unit (three per score), each alone at full rate."""
    clk = sms * mhz
    return {"tensor": pairs * H * 2 * (dk + dv) / tflops / 1e6, "fp32": pairs * (H * H + 8 * H) / 128 / clk,
            "sfu": pairs * 3 * H / 16 / clk}


def kernels(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), hbm_gbs: float = 6547.0,
            tflops: float = 1654.0) -> dict:
    """Every kernel of the family alone: ragged prompts (8 of 1024 tokens), decode at 64 and 256 sequences with
    full windows; beside the prefill / decode attention of the GQA family on the same shapes."""
    dev, dt = torch.device("cuda"), torch.bfloat16
    out = {}
    for name in sizes:
        z = SIZES[name]
        d, H, G, D, (Hr, dk, dv), F, W = z["d"], z["H"], z["G"], z["dim"], z["rec"], z["ff"], z["window"]
        g = torch.Generator(device=dev).manual_seed(1)
        rnd = lambda *s, dtype=dt: torch.randn(*s, generator=g, device=dev, dtype=dtype)
        res = {}
        lens = [1024] * 8
        T, bs, n = sum(lens), 64, len(lens)
        nb = T // bs
        c = ops.TalkingHeads(D ** -0.5, 30.0, torch.rand(H), torch.rand(H), (torch.eye(H) + 0.1 * torch.randn(H, H)).bfloat16(), W, dev)
        kc, vc = rnd(nb, bs, G, D), rnd(nb, bs, G, D)
        bt = torch.randperm(nb, generator=g, device=dev).int().view(n, -1)
        cu = torch.tensor(np.concatenate([[0], np.cumsum(lens)]), dtype=torch.int32, device=dev)
        q, gate = rnd(T, H * D), rnd(T, H * D)
        tp = ops.prefill_plan(cu, T, 1024, ops.TALKING_TILE_ROWS)     # once per step, shared by the layers
        ms = _time(lambda: ops.talking_attention(q, gate, kc, vc, bt, c, cu_seqlens_q=cu, cu_seqlens_k=cu, max_seqlen_q=1024,
                                                 plan=tp),
                   steps, warmup)
        pairs = _visible_pairs(lens, W)
        roof = talking_roofline_us(pairs, H, D, D, tflops)
        flops = pairs * H * 4 * D
        res["prefill_attention"] = dict(us=ms * 1e3, tflops=flops / ms / 1e9, bounds_us=roof,
                                        frac=max(roof.values()) / ms / 1e3, frac_tensor=roof["tensor"] / ms / 1e3)
        k3, v3 = rnd(T, G, D), rnd(T, G, D)
        rows = ops.prefill_tile_rows(H, G, D, D, dt)
        plan = ops.prefill_plan(cu, T, 1024, rows)
        ms = _time(lambda: ops.prefill_varlen(q.view(T, H, D), k3, v3, cu, cu, 1024, 1024, D ** -0.5, plan=plan), steps, warmup)
        res["gqa_prefill_attention"] = dict(us=ms * 1e3, tflops=flops / ms / 1e9, frac_tensor=flops / ms / 1e9 / tflops)
        st = torch.zeros(256, Hr, dk, dv, device=dev)
        sl = torch.arange(256, device=dev)
        proj = rnd(T, 2 * Hr * dk + Hr * dv)
        parts = lambda x: (x[:, :Hr * dk], x[:, Hr * dk:2 * Hr * dk], x[:, 2 * Hr * dk:])
        fb, lo, nw = torch.full((Hr * dk,), 3.0, device=dev), torch.zeros(Hr * dk, device=dev), torch.ones(dv, device=dev)
        ms = _time(lambda: ops.gated_recurrence(*parts(proj), fb, lo, nw, 1e-5, st, sl, cu_seqlens_q=cu, cu_seqlens_k=cu,
                                                max_seqlen_q=1024), steps, warmup)
        fma = T * Hr * dk * dv * 3 / 128 / (148 * 1965.0)       # one pass: forget, write, read
        res["prefill_recurrence"] = dict(us=ms * 1e3, fp32_bound_us=fma, frac=fma / ms / 1e3)
        x, h, nwd = torch.zeros(T, STREAMS, d, device=dev), rnd(T, d), torch.zeros(d, device=dev)
        mix, wv = torch.eye(STREAMS, device=dev), torch.ones(STREAMS, device=dev)
        for kind, y1 in (("streams", None), ("streams_join", rnd(T, d))):
            ms = _time(lambda: ops.stream_update(x, nwd, 1e-5, dt, y=h, y1=y1, join_w=(nwd, nwd) if y1 is not None else None,
                                                 layer_scale=nwd, mix=mix, out_w=wv, in_w=wv), steps, warmup)
            nbytes = T * d * (STREAMS * 8 + 2 + 2 + (2 if y1 is not None else 0))
            res[kind] = dict(us=ms * 1e3, gbs=nbytes / ms / 1e6, frac=nbytes / ms / 1e6 / hbm_gbs)
        a, r = rnd(T, d), rnd(T, d)
        ms = _time(lambda: ops.add_rmsnorm(a, nwd, 1e-5, r), steps, warmup)
        res["add_rmsnorm_of_gqa"] = dict(us=ms * 1e3, gbs=T * d * 8 / ms / 1e6, frac=T * d * 8 / ms / 1e6 / hbm_gbs)
        gu = rnd(T, 2 * F)
        for kind, fn in (("clamped_glu", lambda: ops.clamped_glu(gu, 7.0, 1.702)), ("swiglu_of_gqa", lambda: ops.swiglu(gu))):
            ms = _time(fn, steps, warmup)
            res[kind] = dict(us=ms * 1e3, gbs=T * F * 6 / ms / 1e6, frac=T * F * 6 / ms / 1e6 / hbm_gbs)
        del gu, x, proj, k3, v3
        for B in (64, 256):
            nbk = (W + bs - 1) // bs
            sets = max(1, int(300e6 / (B * W * 2 * G * D * 2)) + 1)     # rotate pools larger than the L2
            kcs, vcs = rnd(sets, B * nbk, bs, G, D), rnd(sets, B * nbk, bs, G, D)
            bts = torch.randperm(B * nbk, generator=g, device=dev).int().view(B, nbk)
            ctx = torch.full((B,), W, dtype=torch.int64, device=dev)
            qd, gd = rnd(B, H * D), rnd(B, H * D)
            it = itertools.count()
            nbytes = B * W * 2 * G * D * 2

            def dec():
                i = next(it) % sets
                ops.talking_attention(qd, gd, kcs[i], vcs[i], bts, c, context_lens=ctx)

            ms = _time(dec, steps * 3, warmup)
            res[f"decode_attention_{B}"] = dict(us=ms * 1e3, gbs=nbytes / ms / 1e6, frac=nbytes / ms / 1e6 / hbm_gbs)
            kc16, vc16 = kcs.view(sets, -1, 16, G, D), vcs.view(sets, -1, 16, G, D)
            bt16 = (bts[:, :, None] * 4 + torch.arange(4, device=dev).int()).reshape(B, -1).contiguous()

            def dec2():
                i = next(it) % sets
                ops.paged_decode_gqa(qd.view(B, H, D), kc16[i], vc16[i], bt16, ctx, D ** -0.5)

            ms = _time(dec2, steps * 3, warmup)
            res[f"gqa_decode_attention_{B}"] = dict(us=ms * 1e3, gbs=nbytes / ms / 1e6, frac=nbytes / ms / 1e6 / hbm_gbs)
            del kcs, vcs, kc16, vc16
            pd = rnd(B, 2 * Hr * dk + Hr * dv)
            sts = torch.zeros(max(1, int(300e6 / (B * Hr * dk * dv * 4)) + 1), B, Hr, dk, dv, device=dev)

            def rec():
                ops.gated_recurrence(*parts(pd), fb, lo, nw, 1e-5, sts[next(it) % sts.shape[0]], sl, context_lens=ctx)

            ms = _time(rec, steps * 3, warmup)
            nbytes = B * Hr * dk * dv * 8
            res[f"decode_recurrence_{B}"] = dict(us=ms * 1e3, gbs=nbytes / ms / 1e6, frac=nbytes / ms / 1e6 / hbm_gbs)
            del sts
        ops.check_status()
        torch.cuda.empty_cache()
        out[name] = res
    return dict(workload="Nabalix kernels alone, bf16", sizes={n: SIZES[n] for n in sizes}, kernels=out)


def engine_rates(cfg: dict, weights, block_size: int, steps: int, warmup: int, batch: int, prompt: int) -> dict:
    """Median wall time of a full prefill step (eight prompts of ``prompt`` tokens) and of a decode step of ``batch``
    sequences, through an engine of its own."""
    from .engine import SamplingParams, Sequence
    from .engine.llm_engine import LLMEngine
    Sequence.counter = itertools.count()
    eng = LLMEngine(dict(model=cfg, weights=weights, dtype=torch.bfloat16, block_size=block_size, max_num_sequences=batch,
                         max_num_batched_tokens=8 * prompt, max_cached_blocks=(batch + 1) * 2 * prompt // block_size, eos=-1,
                         device="cuda:0", max_model_length=2 * prompt, seed=0))
    mixed = getattr(eng.model_runner, "mixed_batches", False)
    rng = np.random.default_rng(0)
    for _ in range(batch):
        eng.add_request(rng.integers(0, VOCAB, size=prompt).tolist(),
                        SamplingParams(temperature=0.0, max_tokens=prompt, ignore_eos=True))
    times = dict(prefill=[], decode=[])
    while len(times["decode"]) < steps + warmup:
        torch.cuda.synchronize()
        t0 = time.perf_counter()
        _, n, is_prefill = eng.step()
        torch.cuda.synchronize()
        if is_prefill and mixed and n != 8 * prompt:
            continue                          # prompts finishing beside decoded tokens
        if not is_prefill and n < batch:
            continue
        times["prefill" if is_prefill else "decode"].append(time.perf_counter() - t0)
    ops.check_status()
    pre, dec = float(np.median(times["prefill"][2:])), float(np.median(times["decode"][warmup:]))
    eng.exit()
    del eng
    torch.cuda.empty_cache()
    return dict(prefill_ms=pre * 1e3, prefill_tokens_per_s=8 * prompt / pre, decode_ms=dec * 1e3,
                decode_tokens_per_s=batch / dec)


def throughput(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), layers: int = 4, batch: int = 64,
               prompt: int = 1024) -> dict:
    """Prefill and decode throughput through the engine: ``layers`` layers of every size, prompts of ``prompt``
    tokens eight to a step, then ``batch`` sequences decoding from captured graphs; the Nabalix model and the GQA
    decoder of the same width, heads, feed-forward and depth."""
    from .model import resolve_config
    from .model.nabalix import init_weights as init_nabalix
    out = {}
    for name in sizes:
        cfg = nabalix_config(SIZES[name], layers)
        # checkpoints of the family hold bf16 values (the head mix then runs on tensor cores)
        a = engine_rates(cfg, init_nabalix(resolve_config(cfg), 0, torch.bfloat16), 64, steps, warmup, batch, prompt)
        b = engine_rates(gqa_config(SIZES[name], layers), None, 16, steps, warmup, batch, prompt)
        out[f"{name}.nabalix"], out[f"{name}.gqa"] = a, b
        out[f"{name}.ratio"] = dict(prefill=a["prefill_tokens_per_s"] / b["prefill_tokens_per_s"],
                                    decode=a["decode_tokens_per_s"] / b["decode_tokens_per_s"])
    return dict(workload=f"engine throughput, {layers} layers, prefill steps of 8 prompts x {prompt} tokens, decode of "
                         f"{batch} sequences with contexts from {prompt}, bf16, random weights", results=out)
