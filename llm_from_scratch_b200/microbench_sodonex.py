"""Timed runs of the Sodonex family: its kernels on layer sizes of real models beside the like kernels of the GQA + MoE decoder, and
prefill / decode throughput of the whole model beside that decoder at equal width, heads, parameters and depth (``bench.py
--workload sodonex`` and ``sodonex_kernels``).  Weights are random; inputs of the kernel runs exceed the L2 or rotate over buffers
that do."""
from __future__ import annotations

import itertools

import numpy as np
import torch

from . import ops
from .microbench_nabalix import VOCAB, _time, engine_rates

# width, heads, kv heads, head size, feed-forward of a SwiGLU expert (a squared-ReLU one is half as wide again: equal parameters),
# experts, experts per token
SIZES = {
    "d1024": dict(d=1024, H=16, G=4, dim=64, ff=1408, E=16, K=2),
    "d2048": dict(d=2048, H=16, G=4, dim=128, ff=1408, E=32, K=4),
    "d4096": dict(d=4096, H=32, G=8, dim=128, ff=2048, E=32, K=4),
}
CHUNK, TAPS = 512, 4


def sodonex_config(z: dict, layers: int, chunk: int = CHUNK) -> dict:
    mixer = dict(heads=z["H"], kv_heads=z["G"], dim=z["dim"], vdim=z["dim"], conv=TAPS, scale=z["dim"] ** -0.5,
                 rot=dict(dims=z["dim"] // 2, base=5e5), mask=dict(size=chunk) if chunk else None)
    mlp = {"kind": "moe", "expert": dict(ff=z["ff"] * 3 // 2), "router": dict(experts=z["E"], top=z["K"])}
    return {"architecture": "Sodonex", "vocab": VOCAB, "width": z["d"], "norm": {"eps": 1e-5}, "embedding": {"scale": 1.0},
            "residual_mult": 0.3, "layers": [{"type": "attention", "mixer": mixer, "mlp": mlp}] * layers}


def gqa_moe_config(z: dict, layers: int) -> dict:
    return dict(vocab_size=VOCAB, context_length=8192, d_model=z["d"], num_layers=layers, num_heads=z["H"], num_kv_heads=z["G"],
                d_ff=z["ff"], attention_type="GQA", use_moe=True, moe_layers=list(range(layers)), n_routed_experts=z["E"],
                num_experts_per_tok=z["K"], n_shared_experts=0)


def _chunk_pairs(lens, chunk: int) -> int:
    """Visible (query, key) pairs of whole prompts."""
    tri = lambda n: n * (n + 1) // 2
    return sum((n // chunk) * tri(chunk) + tri(n % chunk) if chunk else tri(n) for n in lens)


def kernels(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), hbm_gbs: float = 6547.0,
            tflops: float = 1654.0) -> dict:
    """Every kernel of the family alone: ragged prompts (8 of 1024 tokens), decode at 64 and 256 sequences with a full chunk of
    visible keys; each followed by the like kernel of the GQA + MoE decoder (attention: with prompts or contexts as long as a
    chunk, the same pairs)."""
    dev, dt, bs, n = torch.device("cuda"), torch.bfloat16, 64, 8
    out = {}
    for name in sizes:
        z = SIZES[name]
        d, H, G, D, F, E, K = z["d"], z["H"], z["G"], z["dim"], z["ff"] * 3 // 2, z["E"], z["K"]
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

        offsets = lambda lens: torch.tensor(np.concatenate([[0], np.cumsum(lens)]), dtype=torch.int32, device=dev)
        # ---- prompts: attention
        lens = [1024] * n
        T, cu = sum(lens), offsets(lens)
        slots, pos = torch.arange(T, device=dev), torch.arange(T, device=dev) % 1024
        bias, gate = torch.full((H,), -2.0, device=dev), rnd(T, H)
        q, k, v = rnd(T, H, D), rnd(T, G, D), rnd(T, G, D)
        plan = ops.prefill_plan(cu, T, 1024, ops.sigmoid_attention_tile_rows(H, G, D, D, dt))
        rows_gqa = ops.prefill_tile_rows(H, G, D, D, dt)
        for c in (0, CHUNK, 256, 128):
            flops = _chunk_pairs(lens, c) * H * 4 * D
            tensor(f"prefill_attention_c{c}", lambda: ops.sigmoid_attention(q, k, v, cu, cu, 1024, D ** -0.5, bias, c, gate, plan=plan), flops)
            short = [c] * (T // c) if c else lens
            cs, ps = offsets(short), ops.prefill_plan(offsets(short), T, max(short), rows_gqa)
            tensor(f"prefill_attention_c{c}.gqa", lambda: ops.prefill_varlen(q, k, v, cs, cs, max(short), max(short), D ** -0.5, plan=ps), flops)
        # other head sizes run the mma.sync kernel; beside the windowed softmax on it
        h2 = 3 * D // 4
        qs, ks, vs = rnd(T, H, h2), rnd(T, G, h2), rnd(T, G, h2)
        plan64 = ops.prefill_plan(cu, T, 1024, 64)
        flops = _chunk_pairs(lens, 0) * H * 4 * h2
        tensor(f"prefill_attention_dim{h2}", lambda: ops.sigmoid_attention(qs, ks, vs, cu, cu, 1024, 0.1, bias, 0, gate, plan=plan64), flops)
        tensor(f"prefill_attention_dim{h2}.window", lambda: ops.prefill_varlen_window(qs, ks, None, vs, cu, cu, 1024, 0.1, plan=plan64), flops)
        del q, k, v, qs, ks, vs
        # ---- prologue
        Cq, Ck = H * D, G * D
        proj, kc, vc = rnd(T, Cq + Ck + H), rnd(T // bs, bs, G, D), rnd(T // bs, bs, G, D)
        wq, wk = rnd(TAPS, Cq, dtype=torch.float32), rnd(TAPS, Ck, dtype=torch.float32)
        ring, freq = torch.zeros(256, TAPS - 1, Cq + Ck, device=dev), ops.rotary_frequencies(5e5, D // 2, dev)
        sl = torch.arange(256, device=dev)
        rows = ops.StepRows(sl, cu, cu)
        nbytes = T * (H * 2 + G * 5) * D * 2
        mem("conv_norm_rope_store", lambda: ops.conv_norm_rope_store(proj[:, :Cq], proj[:, Cq:Cq + Ck], wq, wk, ring, rows, ones(Cq), ones(Ck),
                                                                     1e-5, freq, pos, kc, vc, slots), nbytes)
        qkv, table = rnd(T, Cq + 2 * Ck), torch.zeros(1024, D, device=dev)
        mem("conv_norm_rope_store.gqa", lambda: ops.qk_norm_rope_store(qkv, ones(Cq), ones(Ck), table, pos, H, G, D, kc, vc, slots), nbytes)
        bt = torch.randperm(T // bs, generator=gen, device=dev).int().view(n, -1)
        ends = torch.arange(n + 1, dtype=torch.int32, device=dev) * 700
        mem("gather_last_rows", lambda: ops.gather_rows(kc.flatten(2), bt, ends, 700, 700 * n, cu), n * 700 * Ck * 4)
        del qkv, proj
        # ---- residual
        x, x2, y, shift, state = torch.zeros(T, d, device=dev), torch.zeros(T, d, device=dev), rnd(T, d), ones(d), torch.zeros(256, d, device=dev)
        move = dict(x_out=x2, shift=shift, state=state, rows=rows)
        mem("residual", lambda: ops.shift_residual(x, 1e-5, dt, x_out=x, y=y, gain=0.3), T * d * 12)
        mem("residual_shift", lambda: ops.shift_residual(x, 1e-5, dt, y=y, gain=0.3, **move), T * d * 12)
        mem("residual_final", lambda: ops.shift_residual(x, 1e-5, dt, y=y, gain=0.3, final_gain=1.0), T * d * 8)
        res2 = rnd(T, d)
        mem("residual.gqa", lambda: ops.add_rmsnorm(y, shift, 1e-5, res2), T * d * 8)
        ey, wts = rnd(T * K, d), torch.rand(T, K, device=dev)
        slot = torch.randperm(T * K, generator=gen, device=dev).int().view(T, K)
        mem("residual_shift_experts", lambda: ops.shift_residual(x, 1e-5, dt, y=ey, gain=0.3, row_weight=wts, slot_to_row=slot, **move),
            T * d * (10 + 2 * K))
        rexp, rw = torch.zeros(T * K, dtype=torch.int32, device=dev), rnd(T * K)
        mem("combine.gqa", lambda: ops.moe_combine(ey, None, rexp, rw, slot), T * d * (2 + 2 * K))
        del ey, res2, x, x2
        # ---- experts
        w_in, w_down, w_gqa = rnd(E, F, d), rnd(E, d, F), rnd(E, 2 * z["ff"], d)
        corr = torch.zeros(E, device=dev)
        for tokens in (64, 256, 2048, 8192):
            logits = rnd(tokens, E, dtype=torch.float32)
            lb = logits.to(dt)
            res[f"route_{tokens}"] = dict(us=_time(lambda: ops.moe_softmax_route(logits, corr, K), steps, warmup) * 1e3)
            res[f"route.gqa_{tokens}"] = dict(us=_time(lambda: ops.moe_route(lb, corr, K), steps, warmup) * 1e3)
            if tokens * K > 256 * E:
                continue
            tok, _, offs, _ = ops.moe_softmax_route(logits, corr, K)
            xs = rnd(tokens, d).index_select(0, tok)
            act = rnd(tokens * K, F)
            hit = int((offs.diff(prepend=offs.new_zeros(1)) > 0).sum())
            for key, fn, width in (("experts_up", lambda: ops.moe_grouped_linear(xs, w_in, offs, squared_relu=True), F),
                                   ("experts_up.gqa", lambda: ops.moe_grouped_gemm(xs, w_gqa, offs, swiglu=True), 2 * z["ff"]),
                                   ("experts_down", lambda: ops.moe_grouped_linear(act, w_down, offs), F),
                                   ("experts_down.gqa", lambda: ops.moe_grouped_gemm(act, w_down, offs), F)):
                if tokens <= 256:
                    mem(f"{key}_{tokens}", fn, hit * d * width * 2)
                else:
                    tensor(f"{key}_{tokens}", fn, tokens * K * d * width * 2)
        del w_in, w_down, w_gqa
        # ---- decode: contexts of two chunks, of which the last one counts; the like kernel has contexts of one chunk
        for B in (64, 256):
            it = itertools.count()
            nbk = 2 * CHUNK // bs
            sets = int(300e6 / (B * CHUNK * 2 * G * D * 2)) + 1                # rotate pools larger than the L2
            kcs, vcs, qd, gd = rnd(sets, B * nbk, bs, G, D), rnd(sets, B * nbk, bs, G, D), rnd(B, H, D), rnd(B, H)
            bts = torch.randperm(B * nbk, generator=gen, device=dev).int().view(B, nbk)
            long, short = (torch.full((B,), c, dtype=torch.int64, device=dev) for c in (2 * CHUNK, CHUNK))
            nbytes = B * CHUNK * 2 * G * D * 2

            def dec():
                i = next(it) % sets
                ops.sigmoid_decode(qd, kcs[i], vcs[i], bts, long, D ** -0.5, bias, CHUNK, gd)

            def dec_gqa():
                i = next(it) % sets
                ops.paged_decode_gqa(qd, kcs[i], vcs[i], bts, short, D ** -0.5)

            mem(f"decode_attention_{B}", dec, nbytes, 3 * steps)
            mem(f"decode_attention.gqa_{B}", dec_gqa, nbytes, 3 * steps)
            del kcs, vcs
            one, pd, pp = ops.StepRows(sl[:B], context_lens=long), rnd(B, Cq + Ck + H), pos[:B]
            res[f"decode_conv_norm_rope_store_{B}"] = dict(us=_time(lambda: ops.conv_norm_rope_store(
                pd[:, :Cq], pd[:, Cq:Cq + Ck], wq, wk, ring, one, ones(Cq), ones(Ck), 1e-5, freq, pp, kc, vc, slots[:B], packed=False),
                steps, warmup) * 1e3)
            qkv = rnd(B, Cq + 2 * Ck)
            res[f"decode_conv_norm_rope_store.gqa_{B}"] = dict(us=_time(lambda: ops.qk_norm_rope_store(
                qkv, ones(Cq), ones(Ck), table, pp, H, G, D, kc, vc, slots[:B]), steps, warmup) * 1e3)
            xd, yd, xo = torch.zeros(B, d, device=dev), rnd(B, d), torch.zeros(B, d, device=dev)
            res[f"decode_residual_shift_{B}"] = dict(us=_time(lambda: ops.shift_residual(
                xd, 1e-5, dt, x_out=xo, y=yd, gain=0.3, shift=shift, state=state, rows=one), steps, warmup) * 1e3)
            res[f"decode_residual.gqa_{B}"] = dict(us=_time(lambda: ops.add_rmsnorm(yd, shift, 1e-5, yd), steps, warmup) * 1e3)
        ops.check_status()
        torch.cuda.empty_cache()
        out[name] = res
    return dict(workload="Sodonex kernels alone, bf16; '.family' rows are the like kernels of other families",
                sizes={n: SIZES[n] for n in sizes}, kernels=out)


def throughput(steps: int = 20, warmup: int = 3, sizes=("d1024", "d2048", "d4096"), layers: int = 4, batch: int = 64,
               prompt: int = 1024) -> dict:
    """Prefill and decode throughput through the engine: ``layers`` layers of every size, prompts of ``prompt`` tokens eight to a
    step, then ``batch`` sequences decoding from captured graphs; beside the GQA + MoE decoder of the same width, heads,
    parameters and depth (full attention, one bf16 residual, SwiGLU experts)."""
    from .model import resolve_config
    from .model.sodonex import init_weights
    out = {}
    for name in sizes:
        cfg = sodonex_config(SIZES[name], layers)
        weights = init_weights(resolve_config(cfg), 0, torch.bfloat16)
        a = engine_rates(cfg, weights, 64, steps, warmup, batch, prompt)
        b = engine_rates(gqa_moe_config(SIZES[name], layers), None, 16, steps, warmup, batch, prompt)
        out[f"{name}.sodonex"], out[f"{name}.gqa"] = a, b
        out[f"{name}.ratio"] = dict(prefill=a["prefill_tokens_per_s"] / b["prefill_tokens_per_s"],
                                    decode=a["decode_tokens_per_s"] / b["decode_tokens_per_s"])
    return dict(workload=f"engine throughput, {layers} layers, chunks of {CHUNK}, prefill steps of 8 prompts x {prompt} tokens, "
                         f"decode of {batch} sequences with contexts from {prompt}, bf16, random weights", results=out)
