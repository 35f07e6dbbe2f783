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

    def __init__(self, parts: list[torch.Tensor], biases: list[torch.Tensor] | None = None):
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
        self.bias = None
        if biases is not None:
            self.bias = torch.zeros(at, dtype=self.weight.dtype, device=self.weight.device)
            for (first, n), b in zip(self.columns, biases):
                self.bias[first:first + n] = b

    def whole(self, x: torch.Tensor) -> torch.Tensor:
        return F.linear(x, self.weight, self.bias)

    def split(self, y: torch.Tensor) -> list[torch.Tensor]:
        return [y[:, at:at + n] for at, n in self.columns]

    def forward(self, x: torch.Tensor) -> list[torch.Tensor]:
        return self.split(self.whole(x))


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


_second_stream: dict = {}       # per device


def side_by_side(first, second, ctx, device):
    """Results of two functions that do not need each other.  A decode step runs the second one on a second CUDA stream: at
    decode sizes neither of the two fills the GPU.  ``second`` returns a tuple of tensors."""
    if ctx.is_prefill:
        return first(), second()
    main = torch.cuda.current_stream()
    side = _second_stream.get(device)
    if side is None:
        side = _second_stream[device] = torch.cuda.Stream(device)
    side.wait_stream(main)
    with torch.cuda.stream(side):
        y1 = second()
    y = first()
    main.wait_stream(side)
    for t in y1:
        t.record_stream(main)      # allocated on the side stream, read on this one
    return y, y1


class ParallelMixer(nn.Module):
    """Two mixers side by side over one input.  Returns both results; their norms and the mean of the two belong
    to the residual update (``join`` holds the norm weights), which the stream kernel does in one pass."""

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
        y, (y1,) = side_by_side(lambda: self.left(*left, ctx), lambda: (self.right(*right, ctx),), ctx, h.device)
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


# ------------------------------------------------------------------------------------------------
# mixers that serve the leading single tokens of a step with their decode kernels (Context.singles / portions)
# ------------------------------------------------------------------------------------------------
def _step_output(x: torch.Tensor, width: int, ctx) -> torch.Tensor:
    """Output rows [T, width] of a step for kernels that write the rows of its sequences; padding rows are zero, so that
    what a later tile loads next to a sequence's last row is finite."""
    out = torch.empty(x.shape[0], width, dtype=x.dtype, device=x.device)
    if ctx.portions is not None and ctx.portions.captured:
        out.zero_()
    elif ctx.portions is not None and ctx.portions.num_tokens < x.shape[0]:
        out[ctx.portions.num_tokens:].zero_()
    elif ctx.portions is None and ctx.singles.rows < x.shape[0]:
        out[ctx.singles.rows:].zero_()
    return out


def _heads(x: torch.Tensor, heads: int, dim: int) -> torch.Tensor:
    """[T, heads * dim] columns of a projection as [T, heads, dim]; a view, also of strided rows."""
    return x.unflatten(1, (heads, dim))


class GatedDeltaRule(nn.Module):
    """Gated delta rule behind a short convolution, with an output norm and a silu gate (``b200_delta_rule`` /
    ``b200_delta_step``); the fp32 state and the convolution's last inputs live in the runner's slot pools."""

    def __init__(self, p: Params, d_model: int, heads: int, kv_heads: int, dim: int, vdim: int, taps: int, eps: float):
        super().__init__()
        sizes = {"q": kv_heads * dim, "k": kv_heads * dim, "v": heads * vdim}
        self.project = FusedProjection([p.lin(n, (w, d_model)) for n, w in sizes.items()]
                                       + [p.lin("g", (heads * vdim, d_model)), p.lin("b", (heads, d_model)),
                                          p.lin("a", (heads, d_model))])
        columns = self.project.columns
        width = columns[3][0]
        conv = torch.zeros(taps, width, device=p.device)
        for (at, n), name in zip(columns, sizes):
            conv[:, at:at + n] = p.f32(name + ".conv", (n, taps)).t()
        self.rule = ops.DeltaRule(heads, kv_heads, dim, vdim, tuple(at for at, _ in columns[:3]), conv,
                                  p.f32("dt_bias", (heads,)), p.f32("A_log", (heads,)), p.f32("norm", (vdim,)), eps)
        self.w_o = p.lin("o", (d_model, heads * vdim))
        self.state = self.conv_ring = torch.empty(0)

    def cache_needs(self):
        c = self.rule
        return [("slot", "state", (c.heads, c.dim, c.vdim)), ("slot", "conv_ring", (c.taps, c.width))]

    def forward(self, h, ctx, positions):
        y = self.project.whole(h)
        _, _, _, g, b, a = self.project.split(y)
        o = _step_output(y, self.rule.heads * self.rule.vdim, ctx)
        if ctx.singles is not None:
            s = ctx.singles
            ops.delta_step(self.rule, y, b, a, g, self.state, self.conv_ring, s.state_slots, s.context_lens, out=o)
        if ctx.portions is not None:
            s = ctx.portions
            ops.delta_rule(self.rule, y, b, a, g, self.state, self.conv_ring, s.state_slots, s.cu_seqlens_q,
                           s.cu_seqlens_k, out=o)
        return F.linear(o, self.w_o)


def _portion_attention(q, k, v, k_cache, v_cache, ctx, scale, out, sink=None):
    """Attention of the step's portions: over the step's own packed keys when every context starts in this step, else
    over the pool."""
    s, H, Hkv, dk, dv = ctx.portions, q.shape[1], v.shape[1], q.shape[2], v.shape[2]
    if s.has_prefix:
        plan = s.plan(ops.prefill_tile_rows(H, Hkv, dk, dv, q.dtype, paged=True))
        ops.prefill_varlen(q, None, None, s.cu_seqlens_q, s.cu_seqlens_k, s.max_seqlen_q, s.max_seqlen_k, scale, k_cache,
                           v_cache, s.block_tables, out=out, plan=plan, sink=sink)
    else:
        plan = s.plan(ops.prefill_tile_rows(H, Hkv, dk, dv, q.dtype))
        ops.prefill_varlen(q, k, v, s.cu_seqlens_q, s.cu_seqlens_q, s.max_seqlen_q, s.max_seqlen_q, scale, out=out, plan=plan,
                           sink=sink)


class SinkAttention(nn.Module):
    """Grouped-query attention with biased projections, a norm per query / key head, interleaved rotation of the first
    channels and a learned sink in the softmax denominator."""

    def __init__(self, p: Params, d_model: int, heads: int, kv_heads: int, dim: int, vdim: int, scale: float, rot_dims: int,
                 rot_base: float, eps: float):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim, self.scale, self.eps = heads, kv_heads, dim, vdim, scale, eps
        sizes = {"q": heads * dim, "k": kv_heads * dim, "v": kv_heads * vdim}
        self.project = FusedProjection([p.lin(n, (w, d_model)) for n, w in sizes.items()],
                                       [p.lin(n + ".b", (w,)) for n, w in sizes.items()])
        self.q_norm, self.k_norm = p.f32("q.norm", (dim,)), p.f32("k.norm", (dim,))
        self.sink = p.f32("sink", (heads,))
        self.freq = ops.rotary_frequencies(rot_base, rot_dims, p.device)
        self.w_o = p.lin("o", (d_model, heads * vdim))
        self.k_cache = self.v_cache = torch.empty(0)

    def cache_needs(self):
        return [("paged", "k_cache", (self.kv_heads, self.dim)), ("paged", "v_cache", (self.kv_heads, self.vdim))]

    def forward(self, h, ctx, positions):
        q, k, v = self.project(h)
        T = h.shape[0]
        q, k = ops.head_norm_rope_store(q, k, v, self.q_norm, self.k_norm, self.eps, self.freq, positions, self.k_cache,
                                        self.v_cache, ctx.slot_mapping)
        o = _step_output(h, self.heads * self.vdim, ctx)
        o3 = o.view(T, self.heads, self.vdim)
        if ctx.singles is not None:
            s = ctx.singles
            ops.paged_decode_gqa(q[:s.rows], self.k_cache, self.v_cache, s.block_tables, s.context_lens, self.scale,
                                 out=o3[:s.rows], sink=self.sink)
        if ctx.portions is not None:
            _portion_attention(q, k, _heads(v, self.kv_heads, self.vdim), self.k_cache, self.v_cache, ctx, self.scale, o3, self.sink)
        return F.linear(o, self.w_o)


class LatentAttention(nn.Module):
    """Attention over cached latent rows without positions, with an output gate.  Single tokens attend in the absorbed
    form (queries and results pass through W_uk / W_uv, keys and values are the latent rows themselves); portions expand
    the rows of their contexts.  ``source``: another layer whose latent rows this one reads instead of its own."""

    def __init__(self, p: Params, d_model: int, heads: int, dim: int, vdim: int, kv_rank: int, scale: float, eps: float,
                 source: "LatentAttention | None" = None):
        super().__init__()
        self.heads, self.dim, self.vdim, self.rank, self.scale, self.eps = heads, dim, vdim, kv_rank, scale, eps
        parts = [p.lin("q", (heads * dim, d_model)), p.lin("g", (heads * vdim, d_model))]
        self.source = [source] if source is not None else []         # in a list: not a submodule of this layer
        if source is None:
            parts.append(p.lin("dkv", (kv_rank, d_model)))
            self.norm = p.f32("dkv.norm", (kv_rank,))
        elif source.source or source.rank != kv_rank:
            raise ValueError("a layer can share the latent rows of a layer that has its own, of the same rank")
        self.project = FusedProjection(parts)
        uk, uv = p.lin("uk", (heads * dim, kv_rank)), p.lin("uv", (heads * vdim, kv_rank))
        self.expand = FusedProjection([uk, uv])
        self.w_uk = uk.view(heads, dim, kv_rank)
        self.w_uv_t = uv.view(heads, vdim, kv_rank).transpose(1, 2)
        self.w_o = p.lin("o", (d_model, heads * vdim))
        self.latent_cache = torch.empty(0)
        self.step_rows = None            # latent rows of the running step's tokens
        self.context_rows = None         # and of its portions' contexts, when some of those began in an earlier step

    def cache_needs(self):
        return [] if self.source else [("paged", "latent_cache", (self.rank,))]

    def _absorbed(self, q, s, o):
        n, H = s.rows, self.heads
        owner = self.source[0] if self.source else self
        q_abs = torch.empty(n, H, self.rank, dtype=q.dtype, device=q.device)
        q3 = _heads(q, H, self.dim)[:n]
        torch.bmm(q3.transpose(0, 1), self.w_uk, out=q_abs.transpose(0, 1))
        lat = ops.mla_decode(q_abs, None, owner.latent_cache, s.block_tables, s.context_lens, self.scale)
        torch.bmm(lat.transpose(0, 1), self.w_uv_t, out=o[:n].view(n, H, self.vdim).transpose(0, 1))

    def _expanded(self, q, ctx, o):
        s, H = ctx.portions, self.heads
        owner = self.source[0] if self.source else self
        rows, cu_k, max_k = owner.step_rows, s.cu_seqlens_q, s.max_seqlen_q
        if s.has_prefix:
            if owner.context_rows is None:
                owner.context_rows = ops.gather_rows(owner.latent_cache, s.block_tables, s.cu_seqlens_k, s.max_seqlen_k, s.total_k)
            rows, cu_k, max_k = owner.context_rows, s.cu_seqlens_k, s.max_seqlen_k
        k, v = self.expand(rows)
        ops.prefill_varlen(_heads(q, H, self.dim), _heads(k, H, self.dim), _heads(v, H, self.vdim), s.cu_seqlens_q, cu_k, s.max_seqlen_q,
                           max_k, self.scale, out=o.view(-1, H, self.vdim),
                           plan=s.plan(ops.prefill_tile_rows(H, H, self.dim, self.vdim, q.dtype)))

    def forward(self, h, ctx, positions):
        q, g, *down = self.project(h)
        if down:
            self.step_rows = ops.latent_norm_store(down[0], self.norm, self.eps, self.latent_cache, ctx.slot_mapping)
            self.context_rows = None
        o = _step_output(h, self.heads * self.vdim, ctx)
        if ctx.singles is not None:
            self._absorbed(q, ctx.singles, o)
        if ctx.portions is not None:
            self._expanded(q, ctx, o)
        return F.linear(ops.sigmoid_gate(o, g), self.w_o)


class SquaredReLU(nn.Module):
    """W_down max(W_up h, 0)^2."""

    def __init__(self, p: Params, d_model: int, d_ff: int):
        super().__init__()
        self.w_up, self.w_down = p.lin("up", (d_ff, d_model)), p.lin("down", (d_model, d_ff))

    def forward(self, h, ctx, positions):
        return F.linear(ops.squared_relu(F.linear(h, self.w_up)), self.w_down)


# ------------------------------------------------------------------------------------------------
# sublayers that run side by side on one normed input, with gates on the way into the residual
# ------------------------------------------------------------------------------------------------
class RunCache:
    """The cache of one run of a mixer whose layer may run several times: what the mixer's ``cache_needs`` lists, as
    attributes that the runner fills."""

    def __init__(self, mixer: nn.Module):
        self.mixer = mixer

    def cache_needs(self):
        return self.mixer.cache_needs()


class RotaryLatentAttention(nn.Module):
    """Latent attention with query latents, a rotary key part shared by the heads, a sliding window (0: none) and a sink.
    Single tokens attend in the absorbed form over the cached rows [latent | rotated part]; portions expand the rows that
    their windows reach.  The caller projects (``projections``: query and key / value down-projection)."""

    def __init__(self, p: Params, d_model: int, heads: int, dim: int, rot_dim: int, vdim: int, q_rank: int, kv_rank: int,
                 scale: float, rotation: ops.Rotation, window: int, eps: float):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim, self.rank = heads, dim, rot_dim, vdim, kv_rank
        self.scale, self.rotation, self.window, self.eps = scale, rotation, window, eps
        self.projections = [p.lin("dq", (q_rank, d_model)), p.lin("dkv", (kv_rank + rot_dim, d_model))]
        self.q_norm, self.kv_norm = p.f32("dq.norm", (q_rank,)), p.f32("dkv.norm", (kv_rank,))
        self.w_uq = p.lin("uq", (heads * (dim + rot_dim), q_rank))
        uk, uv = p.lin("uk", (heads * dim, kv_rank)), p.lin("uv", (heads * vdim, kv_rank))
        self.expand = FusedProjection([uk, uv])
        self.w_uk = uk.view(heads, dim, kv_rank)
        self.w_uv_t = uv.view(heads, vdim, kv_rank).transpose(1, 2)
        self.sink = p.f32("sink", (heads,))
        self.w_o = p.lin("o", (d_model, heads * vdim))

    def cache_needs(self):
        return [("paged", "latent_cache", (self.rank + self.rot_dim,))]

    def tile_rows(self, dtype) -> int:
        """Query rows per tile of the kernel that serves this layer's portions; 0: a general one without tile lists."""
        return ops.prefill_window_tile_rows(self.heads, self.heads, self.dim + self.rot_dim, self.rot_dim, self.vdim, dtype)

    row_multiple = 8      # single tokens of mixed steps: the batched products meet few distinct sizes (cf. prefill_token_multiple)
    key_multiple = 256    # the same for the rows of contexts that are expanded

    def _absorbed(self, q, q_rot, cache, ctx, o):
        s, H = ctx.singles, self.heads
        n = m = s.rows
        if ctx.portions is not None and -(-n // self.row_multiple) * self.row_multiple <= ctx.portions.num_tokens:
            m = -(-n // self.row_multiple) * self.row_multiple     # rows n .. m - 1 are of portions, which write them later
        q_abs, lat = (torch.empty(m, H, self.rank, dtype=q.dtype, device=q.device) for _ in range(2))
        torch.bmm(q[:m, :, :self.dim].transpose(0, 1), self.w_uk, out=q_abs.transpose(0, 1))
        ops.mla_decode(q_abs[:n], q_rot, cache, s.block_tables, s.context_lens, self.scale, out=lat[:n], window=self.window,
                       sink=self.sink)
        torch.bmm(lat.transpose(0, 1), self.w_uv_t, out=o[:m].view(m, H, self.vdim).transpose(0, 1))

    def _expanded(self, q, rows, cache, s, o):
        H, keys = self.heads, s.keys(self.window)
        cu_k = s.cu_seqlens_q
        if keys.has_prefix:
            cu_k = keys.cu_seqlens_k
            rows = ops.gather_rows(cache, s.block_tables, cu_k, keys.max_seqlen_k, keys.total_k, s.cu_seqlens_k,
                                   self.key_multiple)
        k, v = self.expand(rows[:, :self.rank])
        k_tail = rows[:, self.rank:] if self.rot_dim else None
        plan = s.plan(self.tile_rows(q.dtype))
        ops.prefill_varlen_window(q, _heads(k, H, self.dim), k_tail, _heads(v, H, self.vdim), s.cu_seqlens_q, cu_k, s.max_seqlen_q,
                                  self.scale, self.window, self.sink, out=o.view(-1, H, self.vdim), plan=plan)

    def forward(self, dq, dkv, ctx, positions, pools):
        c_q, rows = ops.latent_prologue(dq, self.q_norm, dkv, self.kv_norm, self.eps, self.rotation, positions,
                                        pools.latent_cache, ctx.slot_mapping)
        q = _heads(F.linear(c_q, self.w_uq), self.heads, self.dim + self.rot_dim)
        singles = ctx.singles.rows if ctx.singles is not None else 0
        q_rot = ops.rotate_heads(q, self.rot_dim, self.rotation, positions, singles) if self.rot_dim else None
        o = _step_output(rows, self.heads * self.vdim, ctx)
        if ctx.singles is not None:
            self._absorbed(q, q_rot, pools.latent_cache, ctx, o)
        if ctx.portions is not None:
            self._expanded(q, rows, pools.latent_cache, ctx.portions, o)
        return F.linear(o, self.w_o)


class PolyNormMLP(nn.Module):
    """W_down (c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3) with z = W_up h.  The caller projects up (``projections``)."""

    def __init__(self, p: Params, d_model: int, d_ff: int, eps: float):
        super().__init__()
        self.eps = eps
        self.projections = [p.lin("up", (d_ff, d_model))]
        self.coef = p.f32("act", (4,))
        self.w_down = p.lin("down", (d_model, d_ff))

    def forward(self, h, up):
        return (F.linear(ops.poly_norm(up, self.coef, self.eps), self.w_down),)


class RoutedExperts(nn.Module):
    """Feed-forwards of which a router picks some per token.  Returns the chosen experts' output rows, their weights and where
    a token's rows are; the weighted sum belongs to the residual update.  A kind of experts says how it routes (``route``), what
    its first map does (``first``) and the same activation behind a plain product (``activation``)."""

    # average rows per expert above which bf16 goes to the library's grouped GEMM (see transformer.MoE)
    own_gemm_max_rows_per_expert = 256

    def __init__(self, p: Params, d_model: int, d_ff: int, experts: int, maps_in: tuple[str, ...]):
        super().__init__()
        self.router = p.lin("router", (experts, d_model))
        self.w_in = torch.stack([torch.cat([p.lin(f"e{e}.{m}", (d_ff, d_model)) for m in maps_in]) for e in range(experts)])
        self.w_down = torch.stack([p.lin(f"e{e}.down", (d_model, d_ff)) for e in range(experts)])
        self.library = p.dtype == torch.bfloat16 and d_model % 8 == 0 and d_ff % 8 == 0

    def forward(self, h):
        z = F.linear(h, self.router) if h.dtype == torch.float32 else torch.mm(h, self.router.t(), out_dtype=torch.float32)
        tok, weight, offs, slot = self.route(z)
        xs = h.index_select(0, tok)
        if self.library and tok.numel() > self.own_gemm_max_rows_per_expert * self.router.shape[0]:
            act = self.activation(torch._grouped_mm(xs, self.w_in.transpose(1, 2), offs=offs))
            return torch._grouped_mm(act, self.w_down.transpose(1, 2), offs=offs), weight, slot
        return ops.moe_grouped_linear(self.first(xs, offs), self.w_down, offs, early_launch=True), weight, slot


class GroupedMoE(RoutedExperts):
    """Clamped GLU experts behind a sigmoid router with a choice correction and groups of experts."""

    def __init__(self, p: Params, d_model: int, d_ff: int, experts: int, top: int, groups: int, keep: int, limit: float,
                 slope: float = 1.702):
        super().__init__(p, d_model, d_ff, experts, ("gate", "up"))
        self.top, self.groups, self.keep, self.limit, self.slope = top, groups, keep, limit, slope
        self.projections = []
        self.correction = p.f32("correction", (experts,))

    def route(self, z):
        return ops.moe_group_route(z, self.correction, self.top, self.groups, self.keep)

    def first(self, xs, offs):
        return ops.moe_grouped_linear(xs, self.w_in, offs, glu=(self.limit, self.slope), early_launch=True)

    def activation(self, h):
        return ops.clamped_glu(h, self.limit, self.slope)


class SoftmaxMoE(RoutedExperts):
    """Squared-ReLU experts behind a router with a bias; the weights are the softmax over the chosen logits."""

    def __init__(self, p: Params, d_model: int, d_ff: int, experts: int, top: int):
        super().__init__(p, d_model, d_ff, experts, ("up",))
        self.top = top
        self.router_bias = p.f32("router.b", (experts,))

    def route(self, z):
        return ops.moe_softmax_route(z, self.router_bias, self.top)

    def first(self, xs, offs):
        return ops.moe_grouped_linear(xs, self.w_in, offs, squared_relu=True, early_launch=True)

    def activation(self, h):
        return ops.squared_relu(h)


class TokenInput(nn.Module):
    """proj (gelu(gate x) * e) with e a part of the token's row in a table that all layers share; the norm of the result
    (``norm``) belongs to the residual update."""

    def __init__(self, p: Params, d_model: int, table: torch.Tensor, first: int, dim: int):
        super().__init__()
        self.table, self.first = table, first
        self.gate, self.proj = p.lin("gate", (dim, d_model)), p.lin("proj", (d_model, dim))
        self.norm = p.f32("norm", (d_model,))

    def forward(self, x, tokens):
        return F.linear(ops.gelu_table(F.linear(x, self.gate), self.table, self.first, tokens), self.proj)


class GatedSublayers(nn.Module):
    """A mixer and (optionally) a feed-forward side by side on the same normed input; every result passes a gate
    sigmoid(W h + b) on its way into the residual.  All linear maps of that input are one GEMM."""

    def __init__(self, p: Params, d_model: int, mixer: nn.Module, mlp: nn.Module | None):
        super().__init__()
        self.mixer, self.mlp = mixer, mlp
        gates = ["rg1"] + (["rg2"] if mlp is not None else [])
        inner = mixer.projections + (mlp.projections if mlp is not None else [])
        self.num_mixer, self.num_inner = len(mixer.projections), len(inner)
        zeros = [torch.zeros(w.shape[0], dtype=w.dtype, device=w.device) for w in inner]
        self.project = FusedProjection(inner + [p.lin(g, (d_model, d_model)) for g in gates],
                                       zeros + [p.lin(g + ".b", (d_model,)) for g in gates])
        mixer.projections = None                       # the fused copy is the one that is kept
        if mlp is not None:
            mlp.projections = None

    def forward(self, h, x, ctx, positions, pools):
        """Adds both sublayers' results to the residual x; returns x in the dtype of h."""
        parts = self.project(h)
        into_mixer, into_mlp, gates = parts[:self.num_mixer], parts[self.num_mixer:self.num_inner], parts[self.num_inner:]
        mix = lambda: self.mixer(*into_mixer, ctx, positions, pools)
        if self.mlp is None:
            return ops.gated_residual(x, mix(), gates[0])
        y, (f, *choice) = side_by_side(mix, lambda: self.mlp(h, *into_mlp), ctx, h.device)
        return ops.gated_residual(x, y, gates[0], f, gates[1], *choice)


# ------------------------------------------------------------------------------------------------
# tokens that look at the ones just before them: shifted inputs, convolved queries and keys
# ------------------------------------------------------------------------------------------------
class TokenShift(nn.Module):
    """Mixes what a mixer reads with the previous token's, channel by channel; the residual kernel does it on the way
    (``ops.shift_residual``), the last token of every sequence lives in the runner's slot pool."""

    def __init__(self, p: Params, d_model: int):
        super().__init__()
        self.weight = p.f32("shift", (d_model,))
        self.state = torch.empty(0)

    def cache_needs(self):
        return [("slot", "state", (self.weight.numel(),))]


class SigmoidAttention(nn.Module):
    """Grouped-query attention whose weights are sigmoid(scale q.k + bias of the head), summed without a normalisation over the
    keys of the query's chunk of positions (0: no chunks).  Queries and keys pass a short causal convolution, then a norm over
    the whole projection and a rotation of channel halves; the values are the convolved keys.  A gate per head follows."""

    def __init__(self, p: Params, d_model: int, heads: int, kv_heads: int, dim: int, taps: int, scale: float, rot_dims: int,
                 rot_base: float, chunk: int, eps: float):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.taps = heads, kv_heads, dim, taps
        self.scale, self.chunk, self.eps = scale, chunk, eps
        sizes = {"q": heads * dim, "k": kv_heads * dim}
        gate = p.lin("g", (heads, d_model))
        self.project = FusedProjection([p.lin(n, (w, d_model)) for n, w in sizes.items()] + [gate],
                                       [p.lin(n + ".b", (w,)) for n, w in sizes.items()] + [gate.new_zeros(heads)])
        self.conv_q, self.conv_k = (p.f32(n + ".conv", (w, taps)).t().contiguous() for n, w in sizes.items())
        self.q_norm, self.k_norm = (p.f32(n + ".norm", (w,)) for n, w in sizes.items())
        self.bias = p.f32("pb", (heads,))
        self.freq = ops.rotary_frequencies(rot_base, rot_dims, p.device)
        self.w_o, self.b_o = p.lin("o", (d_model, heads * dim)), p.lin("o.b", (d_model,))
        self.k_cache = self.v_cache = torch.empty(0)
        self.conv_ring = None                              # one tap: nothing is carried over

    def cache_needs(self):
        row = (self.kv_heads, self.dim)
        needs = [("paged", "k_cache", row), ("paged", "v_cache", row)]
        if self.taps > 1:
            needs.append(("slot", "conv_ring", (self.taps - 1, (self.heads + self.kv_heads) * self.dim)))
        return needs

    def tile_rows(self, dtype) -> int:
        """Query rows per tile of the kernel that serves this layer's portions; 0: a general one without tile lists."""
        return ops.sigmoid_attention_tile_rows(self.heads, self.kv_heads, self.dim, self.dim, dtype)

    def _portions(self, q, k, v, gate, s, out):
        keys, cu_k = s.keys(chunk=self.chunk), s.cu_seqlens_q
        if keys.has_prefix:
            cu_k = keys.cu_seqlens_k
            k, v = (ops.gather_rows(c.flatten(2), s.block_tables, cu_k, keys.max_seqlen_k, keys.total_k,
                                    s.cu_seqlens_k).unflatten(1, (self.kv_heads, self.dim)) for c in (self.k_cache, self.v_cache))
        ops.sigmoid_attention(q, k, v, s.cu_seqlens_q, cu_k, s.max_seqlen_q, self.scale, self.bias, self.chunk, gate, out=out,
                              plan=s.plan(self.tile_rows(q.dtype)))

    def forward(self, h, ctx, positions, rows):
        q, k, gate = self.project(h)
        q, k, v = ops.conv_norm_rope_store(q, k, self.conv_q, self.conv_k, self.conv_ring, rows, self.q_norm, self.k_norm, self.eps,
                                           self.freq, positions, self.k_cache, self.v_cache, ctx.slot_mapping,
                                           packed=ctx.portions is not None)
        o = _step_output(h, self.heads * self.dim, ctx)
        o3 = o.view(-1, self.heads, self.dim)
        if ctx.singles is not None:
            s = ctx.singles
            ops.sigmoid_decode(q[:s.rows], self.k_cache, self.v_cache, s.block_tables, s.context_lens, self.scale, self.bias,
                               self.chunk, gate[:s.rows], out=o3[:s.rows])
        if ctx.portions is not None:
            self._portions(q, k, v, gate, ctx.portions, o3)
        return F.linear(o, self.w_o, self.b_o)
