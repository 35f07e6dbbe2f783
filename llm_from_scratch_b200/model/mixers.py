"""Token mixers and feed-forwards that decoder families compose (beside the GQA / MLA layers of ``transformer``).

Every class takes its sizes and constants as arguments and its weights from a ``Params`` view, reads the step's
``Context`` and leaves the caching to the runner: a mixer declares the pools it needs through ``cache_needs`` and
finds them as attributes when it runs.  Mixers that read the same input share one projection GEMM: each gives
its linear weights to a ``FusedProjection`` and picks its columns from the result.
"""
from __future__ import annotations

import torch
import torch.nn.functional as F
from torch import nn

from .. import ops


class Params:
    """Named CPU weights on their way to the device: ``lin`` in the compute dtype, ``f32`` in fp32."""

    def __init__(self, weights: dict, device, dtype, prefix: str = ""):
        self.w, self.device, self.dtype, self.prefix = weights, device, dtype, prefix

    def at(self, prefix: str) -> "Params":
        return Params(self.w, self.device, self.dtype, self.prefix + prefix)

    def __contains__(self, name: str) -> bool:
        return self.prefix + name in self.w

    def raw(self, name: str, shape=None) -> torch.Tensor:
        t = self.w.get(self.prefix + name)
        if t is None:
            raise KeyError(f"checkpoint lacks {self.prefix + name}")
        if shape is not None and tuple(t.shape) != tuple(shape):
            raise ValueError(f"shape mismatch for {self.prefix + name}: checkpoint {tuple(t.shape)}, model {tuple(shape)}")
        return t

    def lin(self, name: str, shape) -> torch.Tensor:
        return self.raw(name, shape).to(self.device, self.dtype).contiguous()

    def f32(self, name: str, shape) -> torch.Tensor:
        return self.raw(name, shape).to(self.device, torch.float32).contiguous()


class FusedProjection(nn.Module):
    """One GEMM for several linear maps of the same input.  Every part starts at a column that is a multiple of
    eight (zero rows in between), so that the kernels behind it can use 16-byte accesses."""

    align = 8

    def __init__(self, parts: list[torch.Tensor]):
        super().__init__()
        rows, self.columns, at = [], [], 0
        for w in parts:
            self.columns.append((at, w.shape[0]))
            rows.append(w)
            pad = -w.shape[0] % self.align
            if pad:
                rows.append(torch.zeros(pad, w.shape[1], dtype=w.dtype, device=w.device))
            at += w.shape[0] + pad
        self.weight = torch.cat(rows).contiguous()

    def forward(self, x: torch.Tensor) -> list[torch.Tensor]:
        y = F.linear(x, self.weight)
        return [y[:, at:at + n] for at, n in self.columns]


class TalkingHeadsAttention(nn.Module):
    """Grouped-query attention without rotation whose heads are mixed before the softmax, with a soft cap, a
    logarithmic distance bias, a sliding window and an output gate (``b200_talking_attention``)."""

    def __init__(self, p: Params, d_model: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float,
                 softcap: float, window: int):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = heads, kv_heads, dim, vdim
        self.consts = ops.TalkingHeads(scale, softcap, p.raw("r1", (heads,)), p.raw("r2", (heads,)),
                                       p.raw("talk", (heads, heads)), window, p.device)
        self.projections = [p.lin("q", (heads * dim, d_model)), p.lin("k", (kv_heads * dim, d_model)),
                            p.lin("v", (kv_heads * vdim, d_model)), p.lin("g", (heads * vdim, d_model))]
        self.w_o = p.lin("o", (d_model, heads * vdim))
        self.k_cache = self.v_cache = torch.empty(0)       # views into the pool, set by the runner

    def cache_needs(self):
        return [("paged", "k_cache", (self.kv_heads, self.dim)), ("paged", "v_cache", (self.kv_heads, self.vdim))]

    def forward(self, q, k, v, g, ctx):
        ops.store_kv_rows(k, v, self.k_cache, self.v_cache, ctx.slot_mapping)
        if ctx.is_prefill:
            o = ops.talking_attention(q, g, self.k_cache, self.v_cache, ctx.block_tables, self.consts,
                                      cu_seqlens_q=ctx.cu_seqlens_q, cu_seqlens_k=ctx.cu_seqlens_k,
                                      max_seqlen_q=ctx.max_seqlen_q, plan=ctx.prefill_plan)
        else:
            o = ops.talking_attention(q, g, self.k_cache, self.v_cache, ctx.block_tables, self.consts,
                                      context_lens=ctx.context_lens)
        return F.linear(o.view(o.shape[0], -1), self.w_o)


class GatedRecurrence(nn.Module):
    """HGRN2 linear attention: the forget gate decides what is kept and what is written
    (``b200_gated_recurrence``); the fp32 state of every sequence lives in the runner's slot pool."""

    def __init__(self, p: Params, d_model: int, heads: int, dim: int, vdim: int, eps: float):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps = heads, dim, vdim, eps
        self.projections = [p.lin("q", (heads * dim, d_model)), p.lin("f", (heads * dim, d_model)),
                            p.lin("v", (heads * vdim, d_model))]
        self.f_bias, self.lower = p.f32("f.b", (heads * dim,)), p.f32("lower", (heads * dim,))
        self.norm = p.f32("norm", (vdim,))
        self.w_o = p.lin("o", (d_model, heads * vdim))
        self.state = torch.empty(0)

    def cache_needs(self):
        return [("slot", "state", (self.heads, self.dim, self.vdim))]

    def forward(self, q, f, v, ctx):
        if ctx.is_prefill:
            o = ops.gated_recurrence(q, f, v, self.f_bias, self.lower, self.norm, self.eps, self.state, ctx.state_slots,
                                     cu_seqlens_q=ctx.cu_seqlens_q, cu_seqlens_k=ctx.cu_seqlens_k,
                                     max_seqlen_q=ctx.max_seqlen_q)
        else:
            o = ops.gated_recurrence(q, f, v, self.f_bias, self.lower, self.norm, self.eps, self.state, ctx.state_slots,
                                     context_lens=ctx.context_lens)
        return F.linear(o, self.w_o)


class ParallelMixer(nn.Module):
    """Two mixers side by side over one input.  Returns both results; their norms and the mean of the two belong
    to the residual update (``join`` holds the norm weights), which the stream kernel does in one pass.

    A decode step runs the right mixer on a second CUDA stream: at decode sizes neither of the two fills the GPU."""

    _side: dict = {}       # second stream per device

    def __init__(self, p: Params, d_model: int, left: nn.Module, right: nn.Module):
        super().__init__()
        self.left, self.right = left, right
        self.project = FusedProjection(left.projections + right.projections)
        self.num_left = len(left.projections)
        left.projections = right.projections = None        # the fused copy is the one that is kept
        self.join = (p.f32("left.out", (d_model,)), p.f32("right.out", (d_model,)))

    def forward(self, h, ctx):
        parts = self.project(h)
        left, right = parts[:self.num_left], parts[self.num_left:]
        if ctx.is_prefill:
            return self.left(*left, ctx), self.right(*right, ctx)
        main = torch.cuda.current_stream()
        side = self._side.setdefault(h.device, None) or torch.cuda.Stream(h.device)
        self._side[h.device] = side
        side.wait_stream(main)
        with torch.cuda.stream(side):
            y1 = self.right(*right, ctx)
        y = self.left(*left, ctx)
        main.wait_stream(side)
        y1.record_stream(main)      # allocated on the side stream, read on this one
        return y, y1


class ClampedGLU(nn.Module):
    """W_down [ g sigmoid(slope g) (u + 1) ] with g = min(W_gate h, limit), u = clamp(W_up h, +-limit)."""

    def __init__(self, p: Params, d_model: int, d_ff: int, limit: float, slope: float = 1.702):
        super().__init__()
        self.limit, self.slope = limit, slope
        self.w_in = torch.cat([p.lin("gate", (d_ff, d_model)), p.lin("up", (d_ff, d_model))]).contiguous()
        self.w_down = p.lin("down", (d_model, d_ff))

    def forward(self, h, ctx):
        return F.linear(ops.clamped_glu(F.linear(h, self.w_in), self.limit, self.slope), self.w_down), None


class HyperConnection(nn.Module):
    """Weights that connect one sublayer to the residual streams: read [S], mix [S, S] (from, to), write [S], plus
    the sublayer's input norm and layer scale."""

    def __init__(self, p: Params, q: int, d_model: int, streams: int):
        super().__init__()
        self.norm = p.f32(f"norm{q}", (d_model,))
        self.scale = p.f32(f"ls{q}", (d_model,))
        self.read = p.f32(f"hc{q}.in", (streams,))
        self.mix = p.f32(f"hc{q}.mix", (streams, streams))
        self.write = p.f32(f"hc{q}.out", (streams,))
