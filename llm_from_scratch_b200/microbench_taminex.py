"""Timed runs of the Taminex family: its kernels on layer sizes of real models beside the like kernels of the other
families, and prefill / decode throughput of the whole model beside the GQA decoder of equal width, heads, parameters
and depth (``bench.py --workload taminex`` and ``taminex_kernels``).  Weights are random; inputs of the kernel runs exceed
the L2 or rotate over buffers that do."""
from __future__ import annotations

import itertools

import numpy as np
import torch

from . import ops
from .microbench_nabalix import _time, _visible_pairs, engine_rates, gqa_config

# width, heads x size of both attentions, latent rank, delta (value heads, key heads, size), feed-forward of the GQA decoder;
# the squared-ReLU feed-forward is half as wide again (equal parameters)
SIZES = {
    "d1024": dict(d=1024, H=16, G=4, dim=64, rank=256, delta=(8, 4, 64), ff=2816),
    "d2048": dict(d=2048, H=16, G=4, dim=128, rank=512, delta=(16, 8, 128), ff=5632),
    "d4096": dict(d=4096, H=32, G=8, dim=128, rank=512, delta=(32, 16, 128), ff=11264),
}
VOCAB, TAPS = 32000, 4


def taminex_config(size: dict, layers: int) -> dict:
    (Hd, Gd, dd), H, dim = size["delta"], size["H"], size["dim"]
    mlp = {"kind": "dense", "ff": size["ff"] * 3 // 2}
    delta = {"type": "delta", "mixer": dict(heads=Hd, kv_heads=Gd, dim=dd, vdim=dd, conv=TAPS), "mlp": mlp}
    latent = {"type": "latent_attention", "mixer": dict(heads=H, dim=dim, vdim=dim, kv_rank=size["rank"], scale=dim ** -0.5),
              "mlp": mlp}
    attention = {"type": "attention", "mixer": dict(heads=H, kv_heads=size["G"], dim=dim, vdim=dim, scale=dim ** -0.5,
                                                    rot=dict(dims=dim // 2, base=5e5)), "mlp": mlp}
    return {"architecture": "Taminex", "vocab": VOCAB, "width": size["d"], "norm": {"eps": 1e-5}, "logit_scale": 0.5,
            "logit_softcap": 15.0, "layers": list(itertools.islice(itertools.cycle([delta, latent, attention, delta]), layers))}


def kernels(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), hbm_gbs: float = 6547.0,
            tflops: float = 1654.0) -> dict:
    """Every kernel of the family alone: ragged prompts (8 of 1024 tokens), decode at 64 and 256 sequences with contexts of
    1024 tokens; each followed by the like kernel of another family on the same shape."""
    dev, dt, bs, n, ctx_len = torch.device("cuda"), torch.bfloat16, 64, 8, 1024
    sms, mhz = 148, 1965.0
    out = {}
    for name in sizes:
        z = SIZES[name]
        d, H, G, D, r, (Hd, Gd, dd), F = z["d"], z["H"], z["G"], z["dim"], z["rank"], z["delta"], z["ff"]
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

        lens = [1024] * n
        T, nb = sum(lens), sum(lens) // bs
        cu = torch.tensor(np.concatenate([[0], np.cumsum(lens)]), dtype=torch.int32, device=dev)
        slots, pos = torch.arange(T, device=dev), torch.arange(T, device=dev) % 1024
        pairs = _visible_pairs(lens, 1 << 30)
        sink, freq = torch.zeros(H, device=dev), ops.rotary_frequencies(5e5, D // 2, dev)
        # ---- prompts
        q3, k3, v3 = rnd(T, H, D), rnd(T, G, D), rnd(T, G, D)
        plan = ops.prefill_plan(cu, T, 1024, ops.prefill_tile_rows(H, G, D, D, dt))
        for key, s in (("prefill_attention", sink), ("prefill_attention.gqa", None)):
            tensor(key, lambda: ops.prefill_varlen(q3, k3, v3, cu, cu, 1024, 1024, D ** -0.5, plan=plan, sink=s), pairs * H * 4 * D)
        kh, vh = rnd(T, H, D), rnd(T, H, D)
        planh = ops.prefill_plan(cu, T, 1024, ops.prefill_tile_rows(H, H, D, D, dt))
        tensor("prefill_latent_attention", lambda: ops.prefill_varlen(q3, kh, vh, cu, cu, 1024, 1024, D ** -0.5, plan=planh),
               pairs * H * 4 * D)
        if D == 128:
            kt, q192 = rnd(T, 64), rnd(T, H, 192)
            tensor("prefill_latent_attention.mla", lambda: ops.prefill_varlen_shared_tail(q192, kh, kt, vh, cu, cu, 1024, 192 ** -0.5),
                   pairs * H * 2 * (192 + 128))
            del kt, q192
        del kh, vh, q3, k3, v3
        qkv = rnd(T, (H + 2 * G) * D)
        kc, vc = rnd(nb, bs, G, D), rnd(nb, bs, G, D)
        part = lambda x, *w: x.split(w, 1)
        nbytes = T * (H * 2 + G * 5) * D * 2
        mem("head_norm_rope_store", lambda: ops.head_norm_rope_store(*part(qkv, H * D, G * D, G * D), ones(D), ones(D), 1e-5, freq, pos,
                                                                     kc, vc, slots), nbytes)
        table = torch.zeros(1024, D, device=dev)
        mem("head_norm_rope_store.gqa", lambda: ops.qk_norm_rope_store(qkv, ones(H * D), ones(G * D), table, pos, H, G, D, kc, vc, slots),
            nbytes)
        del qkv
        lat = rnd(nb, bs, r)
        proj, w = rnd(T, r), ones(r)
        mem("latent_norm_store", lambda: ops.latent_norm_store(proj, w, 1e-5, lat, slots), T * r * 6)
        bt = torch.randperm(nb, generator=gen, device=dev).int().view(n, -1)
        mem("gather_rows", lambda: ops.gather_rows(lat, bt, cu, 1024, T), T * r * 4)
        o, g2 = rnd(T, H * D), rnd(T, H * D)
        mem("sigmoid_gate", lambda: ops.sigmoid_gate(o, g2), T * H * D * 6)
        x, y, nw = torch.zeros(T, d, device=dev), rnd(T, d), torch.ones(d, device=dev)
        mem("residual_norm", lambda: ops.residual_norm(x, 1e-5, dt, y=y, norm_w=nw), T * d * 12)
        res2 = rnd(T, d)
        mem("residual_norm.gqa", lambda: ops.add_rmsnorm(y, nw, 1e-5, res2), T * d * 8)
        up, gu = rnd(T, F * 3 // 2), rnd(T, 2 * F)
        mem("squared_relu", lambda: ops.squared_relu(up), T * F * 6)
        mem("squared_relu.gqa", lambda: ops.swiglu(gu), T * F * 6)
        del up, gu, o, g2, x, y, res2
        width = (2 * Gd + Hd) * dd
        y = rnd(T, width + Hd * dd + 2 * Hd)
        conv = rnd(TAPS, width, dtype=torch.float32)
        c = ops.DeltaRule(Hd, Gd, dd, dd, (0, Gd * dd, 2 * Gd * dd), conv, torch.zeros(Hd, device=dev) - 2, torch.zeros(Hd, device=dev), ones(dd), 1e-5)
        views = lambda t: (t[:, width + Hd * dd:][:, :Hd], t[:, width + Hd * dd + Hd:], t[:, width:width + Hd * dd])
        st, ring = torch.zeros(256, Hd, dd, dd, device=dev), torch.zeros(256, TAPS, width, device=dev)
        sl = torch.arange(256, device=dev)
        b, a, gate = views(y)
        ms = _time(lambda: ops.delta_rule(c, y, b, a, gate, st, ring, sl, cu, cu), steps, warmup)
        fma = T * Hd * dd * dd * 4 / 128 / (sms * mhz)         # one fp32 pass: decay, read, write, read-out
        res["prefill_delta_rule"] = dict(us=ms * 1e3, fp32_bound_us=fma, frac=fma / ms / 1e3)
        lower, f3 = torch.zeros(Hd * dd, device=dev), torch.full((Hd * dd,), 3.0, device=dev)
        rec = rnd(T, 3 * Hd * dd)
        ms = _time(lambda: ops.gated_recurrence(*part(rec, Hd * dd, Hd * dd, Hd * dd), f3, lower, ones(dd), 1e-5, st, sl,
                                                cu_seqlens_q=cu, cu_seqlens_k=cu, max_seqlen_q=1024), steps, warmup)
        fma = T * Hd * dd * dd * 3 / 128 / (sms * mhz)
        res["prefill_delta_rule.nabalix"] = dict(us=ms * 1e3, fp32_bound_us=fma, frac=fma / ms / 1e3)
        del rec, y
        # ---- decode
        for B in (64, 256):
            nbk, it = ctx_len // bs, itertools.count()
            ctx = torch.full((B,), ctx_len, dtype=torch.int64, device=dev)
            bts = torch.randperm(B * nbk, generator=gen, device=dev).int().view(B, nbk)
            sets = int(300e6 / (B * ctx_len * 2 * G * D * 2)) + 1             # rotate pools larger than the L2
            kcs, vcs, qd = rnd(sets, B * nbk, bs, G, D), rnd(sets, B * nbk, bs, G, D), rnd(B, H, D)
            for key, s in (("decode_attention", sink), ("decode_attention.gqa", None)):
                def dec():
                    i = next(it) % sets
                    ops.paged_decode_gqa(qd, kcs[i], vcs[i], bts, ctx, D ** -0.5, sink=s)
                mem(f"{key}_{B}", dec, B * ctx_len * 2 * G * D * 2, 3 * steps)
            del kcs, vcs
            for key, dr, rr, Hq in (("decode_latent", 0, r, H), ("decode_latent.mla", 64, 512, 16)):
                sets = int(300e6 / (B * ctx_len * (rr + dr) * 2)) + 1
                pool = rnd(sets, B * nbk, bs, rr + dr)
                qa, qr = rnd(B, Hq, rr), rnd(B, Hq, dr) if dr else None

                def lat_dec():
                    ops.mla_decode(qa, qr, pool[next(it) % sets], bts, ctx, 0.05)
                mem(f"{key}_{B}", lat_dec, B * ctx_len * (rr + dr) * 2, 3 * steps)
                del pool
            yd = rnd(B, width + Hd * dd + 2 * Hd)
            b, a, gate = views(yd)
            sets = int(300e6 / (B * Hd * dd * dd * 4)) + 1
            sts, rings = torch.zeros(sets, B, Hd, dd, dd, device=dev), torch.zeros(sets, B, TAPS, width, device=dev)

            def step():
                i = next(it) % sets
                ops.delta_step(c, yd, b, a, gate, sts[i], rings[i], sl, ctx)
            mem(f"decode_delta_{B}", step, B * Hd * dd * dd * 8 + B * width * 4 * TAPS, 3 * steps)
            pd = rnd(B, 3 * Hd * dd)

            def rec_step():
                ops.gated_recurrence(*part(pd, Hd * dd, Hd * dd, Hd * dd), f3, lower, ones(dd), 1e-5, sts[next(it) % sets], sl,
                                     context_lens=ctx)
            mem(f"decode_delta.nabalix_{B}", rec_step, B * Hd * dd * dd * 8, 3 * steps)
            del sts, rings
        logits = rnd(64, VOCAB, dtype=torch.float32)
        mem("softcap_logits", lambda: ops.softcap_logits(logits, 0.5, 15.0), 64 * VOCAB * 8)
        ops.check_status()
        torch.cuda.empty_cache()
        out[name] = res
    return dict(workload="Taminex kernels alone, bf16; '.family' rows are the like kernels of other families",
                sizes={n: SIZES[n] for n in sizes}, kernels=out)


def throughput(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), layers: int = 4, batch: int = 64,
               prompt: int = 1024) -> dict:
    """Prefill and decode throughput through the engine: ``layers`` layers of every size (delta, latent, attention, delta),
    prompts of ``prompt`` tokens eight to a step, then ``batch`` sequences decoding from captured graphs; beside the GQA
    decoder of the same width, heads, parameters and depth."""
    from .model import resolve_config
    from .model.taminex import init_weights
    out = {}
    for name in sizes:
        cfg = taminex_config(SIZES[name], layers)
        weights = init_weights(resolve_config(cfg), 0, torch.bfloat16)
        a = engine_rates(cfg, weights, 64, steps, warmup, batch, prompt)
        b = engine_rates(gqa_config(SIZES[name], layers), None, 16, steps, warmup, batch, prompt)
        out[f"{name}.taminex"], out[f"{name}.gqa"] = a, b
        out[f"{name}.ratio"] = dict(prefill=a["prefill_tokens_per_s"] / b["prefill_tokens_per_s"],
                                    decode=a["decode_tokens_per_s"] / b["decode_tokens_per_s"])
    return dict(workload=f"engine throughput, {layers} layers, prefill steps of 8 prompts x {prompt} tokens, decode of "
                         f"{batch} sequences with contexts from {prompt}, bf16, random weights", results=out)
