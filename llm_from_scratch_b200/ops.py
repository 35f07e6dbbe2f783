"""Tensor-level wrappers over the C ABI: the calls the attention layers of the engine make.

Every function takes CUDA tensors, checks shapes/dtypes on the host, and enqueues the kernel on
the current CUDA stream.  Nothing here computes on the CPU; a CPU tensor is an error.
"""
from __future__ import annotations

import array
import math
from dataclasses import dataclass

import torch

from . import _lib
from ._lib import lib, check

_DTYPES = {torch.float32: _lib.DTYPE_F32, torch.bfloat16: _lib.DTYPE_BF16}

# Epsilon of the reference's q / k / latent RMSNorm layers, nn.RMSNorm(eps=None) (GQA.py:39-40, MLA.py:71-72).
# With fp32 parameters and a bf16 activation (the reference's autocast mode) torch evaluates that layer in
# fp32 with the fp32 machine epsilon and rounds once at the end; in fp32 it is the same number.
VECTOR_NORM_EPS = float(torch.finfo(torch.float32).eps)

_status: dict[int, torch.Tensor] = {}
_workspaces: dict[tuple[int, str], torch.Tensor] = {}
_retired_workspaces: list[torch.Tensor] = []   # outgrown buffers that captured graphs may still address


def _dt(t: torch.Tensor) -> int:
    try:
        return _DTYPES[t.dtype]
    except KeyError:
        raise TypeError(f"unsupported dtype {t.dtype}; the kernels take float32 or bfloat16") from None


def _cuda(*ts: torch.Tensor | None) -> torch.device:
    dev = None
    for t in ts:
        if t is None:
            continue
        if not t.is_cuda:
            raise ValueError("b200 ops take CUDA tensors only (there is no CPU path)")
        if dev is not None and t.device != dev:
            raise ValueError("all tensors must be on the same device")
        dev = t.device
    return dev


def _stream() -> int:
    """The current stream's handle, without building a stream object (an eager step asks for it once per launch)."""
    return torch._C._cuda_getCurrentRawStream(torch._C._cuda_getDevice())


def status_word(device: torch.device) -> torch.Tensor:
    """Per-device int32 that kernels set when they skip an out-of-pool block id or slot."""
    idx = device.index if device.index is not None else torch.cuda.current_device()
    if idx not in _status:
        _status[idx] = torch.zeros(1, dtype=torch.int32, device=device)
    return _status[idx]


def check_status(device: torch.device | None = None) -> None:
    """Synchronises the current stream, raises if a kernel reported a device-side fault."""
    device = device or torch.device("cuda", torch.cuda.current_device())
    st = status_word(device)
    host = array.array("i", [0])
    addr, _ = host.buffer_info()
    check(lib.b200_read_status(st.data_ptr(), addr, _stream()), "read_status")
    if host[0] != 0:
        check(host[0], "device-side check")


def selftest_bounded_wait(poll_limit: int = 1024, device: torch.device | None = None) -> list[int]:
    """Diagnostic: makes a bounded barrier wait run out inside one small CTA (``b200_selftest_bounded_wait``).
    Returns the five result words; the device status word then holds the time-out code, so the next
    ``check_status`` raises (``read_status_code`` reads and clears it without raising)."""
    device = device or torch.device("cuda", torch.cuda.current_device())
    result = torch.full((5,), -1, dtype=torch.int32, device=device)
    check(lib.b200_selftest_bounded_wait(poll_limit, result.data_ptr(), status_word(device).data_ptr(), _stream()),
          "selftest_bounded_wait")
    return result.tolist()


def read_status_code(device: torch.device | None = None) -> int:
    """Synchronises the current stream and returns (and clears) the device status word: 0 or a B200_ERR_* code."""
    device = device or torch.device("cuda", torch.cuda.current_device())
    host = array.array("i", [0])
    addr, _ = host.buffer_info()
    check(lib.b200_read_status(status_word(device).data_ptr(), addr, _stream()), "read_status")
    return host[0]


def workspace(device: torch.device, nbytes: int, tag: str) -> torch.Tensor:
    """Scratch buffer per (device, op); allocated outside any graph capture.

    A captured CUDA graph has the address of the buffer it was captured with baked in, so a buffer
    that has been handed out is never freed: when a later call needs more, a larger one (at least
    twice the size, so all retired buffers together stay below the live one) replaces it for new
    calls and the old one is kept alive for the graphs that still write to it.  Buffers start zero-filled
    (the decode kernels keep arrival counters at the head of theirs, which every call returns to zero);
    nothing else survives a call, so old and new buffers can be in use side by side."""
    idx = device.index if device.index is not None else torch.cuda.current_device()
    key = (idx, tag)
    w = _workspaces.get(key)
    if w is None or w.numel() < nbytes:
        if w is not None:
            _retired_workspaces.append(w)
            nbytes = max(nbytes, 2 * w.numel())
        w = torch.zeros(max(nbytes, 256), dtype=torch.uint8, device=device)
        _workspaces[key] = w
    return w


def store_kvcache(k: torch.Tensor, v: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                  slot_mapping: torch.Tensor) -> None:
    """k_cache[slot_mapping[t]] = k[t], v likewise; slots < 0 are skipped.

    k, v: [T, Hkv, D] (rows contiguous, token stride free); caches: [..., Hkv, D] contiguous.
    """
    dev = _cuda(k, v, k_cache, v_cache, slot_mapping)
    T, Hkv, D = k.shape
    if v.shape != k.shape or k.dtype != v.dtype or k_cache.dtype != k.dtype or v_cache.dtype != k.dtype:
        raise ValueError("k/v/cache shape or dtype mismatch")
    if slot_mapping.dtype != torch.int64 or slot_mapping.numel() != T or not slot_mapping.is_contiguous():
        raise ValueError("slot_mapping must be a contiguous int64 tensor with one entry per token")
    if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise ValueError("caches must be contiguous")
    if k.stride(2) != 1 or k.stride(1) != D or v.stride(2) != 1 or v.stride(1) != D:
        raise ValueError("k/v rows (Hkv*D) must be contiguous")
    if k_cache.shape[-2:] != (Hkv, D) or v_cache.shape != k_cache.shape:
        raise ValueError("cache trailing dims must be (Hkv, D)")
    num_slots = k_cache.numel() // (Hkv * D)
    check(lib.b200_store_kvcache(k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0),
                                 k_cache.data_ptr(), v_cache.data_ptr(), slot_mapping.data_ptr(),
                                 T, Hkv, D, num_slots, _dt(k), status_word(dev).data_ptr(),
                                 _stream()), "store_kvcache")


def store_rows(rows: torch.Tensor, cache: torch.Tensor, slot_mapping: torch.Tensor) -> None:
    """cache[slot_mapping[t]] = rows[t] for a single pool (the MLA latent cache).

    rows: [T, W] with contiguous rows; cache: [..., W] contiguous.
    """
    dev = _cuda(rows, cache, slot_mapping)
    T, W = rows.shape
    if cache.shape[-1] != W or cache.dtype != rows.dtype or not cache.is_contiguous() or rows.stride(1) != 1:
        raise ValueError("rows/cache shape, dtype or layout mismatch")
    if slot_mapping.dtype != torch.int64 or slot_mapping.numel() != T or not slot_mapping.is_contiguous():
        raise ValueError("slot_mapping must be a contiguous int64 tensor with one entry per row")
    check(lib.b200_store_kvcache(rows.data_ptr(), None, rows.stride(0), 0, cache.data_ptr(), None,
                                 slot_mapping.data_ptr(), T, 1, W, cache.numel() // W, _dt(rows),
                                 status_word(dev).data_ptr(), _stream()), "store_rows")


def paged_decode_gqa(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                     block_tables: torch.Tensor, context_lens: torch.Tensor, scale: float,
                     out: torch.Tensor | None = None, sink: torch.Tensor | None = None) -> torch.Tensor:
    """One query token per sequence over a paged KV pool.

    q: [B, Hq, D]; caches: [num_blocks, block_size, Hkv, D] (value heads may have a size of their own);
    block_tables: [B, maxb] int32; context_lens: [B] int64; ``sink`` fp32 [Hq]: exp(sink) joins the softmax
    denominator.  Returns out [B, Hq, Dv].
    """
    dev = _cuda(q, k_cache, v_cache, block_tables, context_lens, out, sink)
    B, Hq, D = q.shape
    nb, bs, Hkv, Dc = k_cache.shape
    Dv = v_cache.shape[3]
    _f32vec("sink", sink, Hq)
    if Dc != D or v_cache.shape[:3] != k_cache.shape[:3] or k_cache.dtype != q.dtype or v_cache.dtype != q.dtype:
        raise ValueError("cache shape/dtype does not match q")
    if block_tables.dtype != torch.int32 or context_lens.dtype != torch.int64:
        raise ValueError("block_tables must be int32 and context_lens int64")
    if block_tables.dim() != 2 or block_tables.shape[0] != B or block_tables.stride(1) != 1:
        raise ValueError("block_tables must be [B, maxb] with contiguous rows")
    if context_lens.numel() != B or not context_lens.is_contiguous():
        raise ValueError("context_lens must be a contiguous [B] tensor")
    if not (q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise ValueError("q and caches must be contiguous")
    if out is None:
        out = torch.empty((B, Hq, Dv), dtype=q.dtype, device=q.device)
    elif out.shape != (B, Hq, Dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [B, Hq, Dv] tensor of q's dtype")
    need = lib.b200_paged_decode_gqa_workspace_bytes(B, Hq, Hkv, D, _dt(q))
    ws = workspace(dev, need, "decode")
    if sink is not None or Dv != D:
        check(lib.b200_paged_decode_sink(q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(),
                                         block_tables.data_ptr(), block_tables.stride(0), context_lens.data_ptr(), B, Hq,
                                         Hkv, D, Dv, bs, nb, float(scale), _ptr(sink), ws.data_ptr(), ws.numel(), _dt(q),
                                         status_word(dev).data_ptr(), _stream()), "paged_decode_sink")
        return out
    check(lib.b200_paged_decode_gqa(q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(),
                                    out.data_ptr(), block_tables.data_ptr(),
                                    block_tables.stride(0), context_lens.data_ptr(), B, Hq, Hkv, D,
                                    bs, nb, float(scale), ws.data_ptr(), ws.numel(), _dt(q),
                                    status_word(dev).data_ptr(), _stream()), "paged_decode_gqa")
    return out


def prefill_varlen(q: torch.Tensor, k: torch.Tensor | None, v: torch.Tensor | None,
                   cu_seqlens_q: torch.Tensor, cu_seqlens_k: torch.Tensor, max_seqlen_q: int,
                   max_seqlen_k: int, scale: float, k_cache: torch.Tensor | None = None,
                   v_cache: torch.Tensor | None = None, block_tables: torch.Tensor | None = None,
                   out: torch.Tensor | None = None, plan: "PrefillPlan | None" = None,
                   slot_mapping: torch.Tensor | None = None, sink: torch.Tensor | None = None) -> torch.Tensor:
    """Causal attention over packed ragged sequences.  ``sink`` (fp32 [Hq]): exp(sink) joins the softmax denominator.

    ``slot_mapping`` (int64, one slot per row of k / v): the same call first scatters the new tokens' k / v
    rows into ``k_cache`` / ``v_cache`` (the step's store_kvcache), with or without ``block_tables``.

    q: [Tq, Hq, Dqk].  Without ``block_tables``: k [Tk, Hkv, Dqk], v [Tk, Hkv, Dv] are the packed
    keys/values.  With ``block_tables`` (a cached prefix exists) keys/values are read from the
    paged caches [num_blocks, block_size, Hkv, D*].  Returns out [Tq, Hq, Dv].  ``plan``: a tile list from
    ``prefill_plan`` for the same ``cu_seqlens_q`` (one CTA per real tile, longest first).
    """
    dev = _cuda(q, k, v, cu_seqlens_q, cu_seqlens_k, k_cache, v_cache, block_tables, out)
    Tq, Hq, Dqk = q.shape
    if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k.dtype != torch.int32:
        raise ValueError("cu_seqlens must be int32")
    num_seqs = cu_seqlens_q.numel() - 1
    if cu_seqlens_k.numel() != num_seqs + 1:
        raise ValueError("cu_seqlens_q and cu_seqlens_k must have the same length")
    if q.stride(2) != 1 or q.stride(1) != Dqk:
        raise ValueError("q heads must be contiguous")
    if block_tables is None:
        if k is None or v is None:
            raise ValueError("k and v are required without block_tables")
        Hkv, Dv = v.shape[1], v.shape[2]
        if k.shape[1] != Hkv or k.shape[2] != Dqk or k.dtype != q.dtype or v.dtype != q.dtype:
            raise ValueError("k/v shape or dtype mismatch")
        if k.stride(2) != 1 or k.stride(1) != Dqk or v.stride(2) != 1 or v.stride(1) != Dv:
            raise ValueError("k/v heads must be contiguous")
        kp, vp, ks, vs = k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0)
        kcp = vcp = btp = 0
        bts = bs = nb = 0
        total_k = k.shape[0]
        if slot_mapping is not None:
            if k_cache is None or v_cache is None or k_cache.shape != v_cache.shape or k_cache.dim() != 4 \
                    or k_cache.shape[2:] != (Hkv, Dqk) or k_cache.dtype != q.dtype \
                    or not (k_cache.is_contiguous() and v_cache.is_contiguous()):
                raise ValueError("the fused scatter needs contiguous caches [num_blocks, block_size, Hkv, D] of q's dtype")
            nb, bs = k_cache.shape[0], k_cache.shape[1]
            kcp, vcp = k_cache.data_ptr(), v_cache.data_ptr()
    else:
        if k_cache is None or v_cache is None:
            raise ValueError("paged prefill needs k_cache and v_cache")
        nb, bs, Hkv, Dk = k_cache.shape
        Dv = v_cache.shape[3]
        if Dk != Dqk or k_cache.dtype != q.dtype or v_cache.dtype != q.dtype:
            raise ValueError("cache shape/dtype does not match q")
        if block_tables.dtype != torch.int32 or block_tables.shape[0] != num_seqs or block_tables.stride(1) != 1:
            raise ValueError("block_tables must be int32 [num_seqs, maxb]")
        if not (k_cache.is_contiguous() and v_cache.is_contiguous()):
            raise ValueError("caches must be contiguous")
        kp = vp = 0
        ks = vs = 0
        total_k = 0
        if slot_mapping is not None:
            if k is None or v is None or k.shape != (Tq, Hkv, Dqk) or v.shape != (Tq, Hkv, Dv) or k.stride(1) != Dqk \
                    or v.stride(1) != Dv or k.stride(2) != 1 or v.stride(2) != 1:
                raise ValueError("the fused scatter needs the new tokens' k / v [Tq, Hkv, D]")
            kp, vp, ks, vs, total_k = k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0), Tq
        kcp, vcp, btp, bts = k_cache.data_ptr(), v_cache.data_ptr(), block_tables.data_ptr(), block_tables.stride(0)
    if slot_mapping is not None and (slot_mapping.dtype != torch.int64 or not slot_mapping.is_contiguous()
                                     or slot_mapping.numel() != min(Tq, total_k)):
        raise ValueError("slot_mapping must be a contiguous int64 tensor with one entry per new token")
    if out is None:
        out = torch.empty((Tq, Hq, Dv), dtype=q.dtype, device=q.device)
    elif out.shape != (Tq, Hq, Dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [Tq, Hq, Dv] tensor")
    args = (q.data_ptr(), kp, vp, out.data_ptr(), q.stride(0), ks, vs, Tq, total_k, cu_seqlens_q.data_ptr(),
            cu_seqlens_k.data_ptr(), num_seqs, int(max_seqlen_q), int(max_seqlen_k), Hq, Hkv, Dqk, Dv, float(scale), kcp,
            vcp, btp, bts, bs, nb, _ptr(slot_mapping), plan.buffer.data_ptr() if plan is not None else None,
            plan.tile_rows if plan is not None else 0, plan.capacity if plan is not None else 0)
    tail = (_dt(q), status_word(dev).data_ptr(), _stream())
    if sink is not None:
        _cuda(q, sink)
        _f32vec("sink", sink, Hq)
        check(lib.b200_prefill_varlen_sink(*args, sink.data_ptr(), *tail), "prefill_varlen_sink")
    else:
        check(lib.b200_prefill_varlen(*args, *tail), "prefill_varlen")
    return out


def prefill_varlen_shared_tail(q: torch.Tensor, k_head: torch.Tensor, k_tail: torch.Tensor, v: torch.Tensor,
                               cu_seqlens_q: torch.Tensor, cu_seqlens_k: torch.Tensor, max_seqlen_q: int,
                               scale: float, out: torch.Tensor | None = None,
                               plan: "PrefillPlan | None" = None) -> torch.Tensor:
    """``prefill_varlen`` over packed keys given in two parts: k_head [Tk, H, Dqk - tail] per head and
    k_tail [Tk, tail], the last columns of every head's key (MLA's shared rotary part).  bf16.

    q: [Tq, H, Dqk], v: [Tk, H, Dv]; token strides are free, heads contiguous.  Returns out [Tq, H, Dv].
    """
    dev = _cuda(q, k_head, k_tail, v, cu_seqlens_q, cu_seqlens_k, out)
    Tq, H, Dqk = q.shape
    Tk, tail = k_tail.shape
    Dv = v.shape[2]
    if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k.dtype != torch.int32 \
            or cu_seqlens_q.numel() != cu_seqlens_k.numel():
        raise ValueError("cu_seqlens must be int32 tensors of the same length")
    if k_head.shape != (Tk, H, Dqk - tail) or v.shape[:2] != (Tk, H):
        raise ValueError("k_head must be [Tk, H, Dqk - tail] and v [Tk, H, Dv]")
    if any(t.dtype != torch.bfloat16 for t in (q, k_head, k_tail, v)):
        raise ValueError("prefill_varlen_shared_tail takes bf16 tensors")
    if q.stride(2) != 1 or q.stride(1) != Dqk or k_head.stride(2) != 1 or k_head.stride(1) != Dqk - tail \
            or v.stride(2) != 1 or v.stride(1) != Dv or k_tail.stride(1) != 1:
        raise ValueError("heads must be contiguous")
    if out is None:
        out = torch.empty((Tq, H, Dv), dtype=q.dtype, device=q.device)
    elif out.shape != (Tq, H, Dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [Tq, H, Dv] tensor")
    check(lib.b200_prefill_varlen_shared_tail(
        q.data_ptr(), k_head.data_ptr(), k_tail.data_ptr(), v.data_ptr(), out.data_ptr(), q.stride(0),
        k_head.stride(0), k_tail.stride(0), v.stride(0), Tq, Tk, cu_seqlens_q.data_ptr(), cu_seqlens_k.data_ptr(),
        cu_seqlens_q.numel() - 1, int(max_seqlen_q), H, Dqk, tail, Dv, float(scale),
        plan.buffer.data_ptr() if plan is not None else None, plan.tile_rows if plan is not None else 0,
        plan.capacity if plan is not None else 0, _dt(q), status_word(dev).data_ptr(), _stream()),
        "prefill_varlen_shared_tail")
    return out


class PrefillPlan:
    """Device-side tile list shared by all prefill attention calls of one step (``prefill_plan``)."""

    __slots__ = ("buffer", "tile_rows", "capacity")

    def __init__(self, buffer: torch.Tensor, tile_rows: int, capacity: int):
        self.buffer, self.tile_rows, self.capacity = buffer, tile_rows, capacity


def prefill_tile_rows(Hq: int, Hkv: int, Dqk: int, Dv: int, dtype: torch.dtype, paged: bool = False) -> int:
    """Query rows per tile of the prefill kernel serving this shape with packed (or ``paged``) keys; 0 = no tiled kernel
    (no plan)."""
    if dtype not in _DTYPES:
        return 0
    if paged and dtype == torch.bfloat16:
        if Dqk == Dv == 128 and Hq // Hkv % 2 == 0:
            return 128                                  # two-head tcgen05 kernel
        return 64 if (Dqk == Dv and Dqk in (32, 64, 128)) or (Dqk, Dv) == (192, 128) else 0
    return int(lib.b200_prefill_tile_rows(Hq, Hkv, Dqk, Dv, _DTYPES[dtype]))


def prefill_plan(cu_seqlens_q: torch.Tensor, total_q_tokens: int, max_seqlen_q: int, tile_rows: int,
                 buffer: torch.Tensor | None = None) -> PrefillPlan | None:
    """Builds the tile list of a prefill step on the device (one small launch).  ``total_q_tokens`` and
    ``max_seqlen_q`` are host-side upper bounds; ``buffer`` (int32) may be supplied to keep the plan
    at a fixed address (graph capture).  Returns None when no tiled kernel applies (tile_rows == 0)."""
    if tile_rows <= 0:
        return None
    dev = _cuda(cu_seqlens_q, buffer)
    if cu_seqlens_q.dtype != torch.int32:
        raise ValueError("cu_seqlens must be int32")
    num_seqs = cu_seqlens_q.numel() - 1
    nbytes = int(lib.b200_prefill_plan_bytes(total_q_tokens, num_seqs, tile_rows))
    if buffer is None:
        buffer = torch.empty(nbytes // 4, dtype=torch.int32, device=dev)
    elif buffer.dtype != torch.int32 or buffer.numel() * 4 < nbytes or not buffer.is_contiguous():
        raise ValueError(f"plan buffer must be contiguous int32 with at least {nbytes // 4} entries")
    check(lib.b200_prefill_plan(cu_seqlens_q.data_ptr(), num_seqs, int(max_seqlen_q), tile_rows, buffer.data_ptr(),
                                buffer.numel() * 4, status_word(dev).data_ptr(), _stream()), "prefill_plan")
    return PrefillPlan(buffer, tile_rows, buffer.numel() - 4)


def mla_decode(q_abs: torch.Tensor, q_rope: torch.Tensor | None, latent_cache: torch.Tensor,
               block_tables: torch.Tensor, context_lens: torch.Tensor, scale: float,
               out: torch.Tensor | None = None, window: int = 0, sink: torch.Tensor | None = None) -> torch.Tensor:
    """Absorbed MLA decode over a paged latent pool.

    q_abs: [B, H, r]; q_rope: [B, H, dr] or None (dr = 0); latent_cache: [num_blocks, block_size, r + dr];
    returns the attention-weighted latent [B, H, r].  ``window`` > 0: over the last ``window`` tokens only; ``sink``
    fp32 [H]: exp(sink) joins the softmax denominator.
    """
    dev = _cuda(q_abs, q_rope, latent_cache, block_tables, context_lens, out, sink)
    B, H, r = q_abs.shape
    _f32vec("sink", sink, H)
    dr = q_rope.shape[2] if q_rope is not None else 0
    nb, bs, row = latent_cache.shape
    if row != r + dr or (q_rope is not None and q_rope.shape[:2] != (B, H)):
        raise ValueError("latent row must be kv_lora_rank + rope_dim wide")
    if latent_cache.dtype != q_abs.dtype or (q_rope is not None and q_rope.dtype != q_abs.dtype):
        raise ValueError("dtype mismatch")
    if block_tables.dtype != torch.int32 or context_lens.dtype != torch.int64:
        raise ValueError("block_tables must be int32 and context_lens int64")
    if block_tables.shape[0] != B or block_tables.stride(1) != 1 or context_lens.numel() != B:
        raise ValueError("metadata batch mismatch")
    if not (q_abs.is_contiguous() and (q_rope is None or q_rope.is_contiguous()) and latent_cache.is_contiguous()):
        raise ValueError("inputs must be contiguous")
    if out is None:
        out = torch.empty_like(q_abs)
    need = lib.b200_mla_decode_workspace_bytes(B, H, r, dr, _dt(q_abs))
    ws = workspace(dev, need, "mla")
    args = (q_abs.data_ptr(), _ptr(q_rope), latent_cache.data_ptr(), out.data_ptr(), block_tables.data_ptr(),
            block_tables.stride(0), context_lens.data_ptr(), B, H, r, dr, bs, nb, float(scale))
    tail = (ws.data_ptr(), ws.numel(), _dt(q_abs), status_word(dev).data_ptr(), _stream())
    if window or sink is not None:
        check(lib.b200_mla_decode_window(*args, int(window), _ptr(sink), *tail), "mla_decode_window")
    else:
        check(lib.b200_mla_decode(*args, *tail), "mla_decode")
    return out


def add_rmsnorm(x: torch.Tensor, weight: torch.Tensor, eps: float, residual: torch.Tensor | None = None):
    """RMSNorm of x (+ residual) in fp32, result in x's dtype.  Returns y, or (y, new_residual) when a
    residual is given (the fused add + norm of the reference's residual stream)."""
    _cuda(x, weight, residual)
    if not x.is_contiguous() or weight.dtype != torch.float32 or weight.numel() != x.shape[-1]:
        raise ValueError("x must be contiguous and weight an fp32 vector of the row width")
    if residual is not None and (residual.shape != x.shape or not residual.is_contiguous()):
        raise ValueError("residual must match x")
    rows, dim = x.numel() // x.shape[-1], x.shape[-1]
    y = torch.empty_like(x)
    res_out = torch.empty_like(x) if residual is not None else None
    check(lib.b200_add_rmsnorm(x.data_ptr(), residual.data_ptr() if residual is not None else None,
                               weight.data_ptr(), y.data_ptr(), res_out.data_ptr() if res_out is not None else None,
                               rows, dim, float(eps), _dt(x), _dt(residual) if residual is not None else 0,
                               _stream()), "add_rmsnorm")
    return y if residual is None else (y, res_out)


def qk_norm_rope_store(qkv: torch.Tensor, q_norm_w: torch.Tensor, k_norm_w: torch.Tensor, rope_table: torch.Tensor,
                       positions: torch.Tensor, num_q_heads: int, num_kv_heads: int, head_dim: int,
                       k_cache: torch.Tensor | None, v_cache: torch.Tensor | None,
                       slot_mapping: torch.Tensor | None):
    """q/k RMSNorm over the whole projected vectors + RoPE + scatter of K/V into the paged cache.

    qkv: [T, (Hq + 2 Hkv) * D] fused projection output; returns (q [T,Hq,D], k [T,Hkv,D], v view [T,Hkv,D]).
    """
    dev = _cuda(qkv, q_norm_w, k_norm_w, rope_table, positions, k_cache, v_cache, slot_mapping)
    T = qkv.shape[0]
    wq, wk = num_q_heads * head_dim, num_kv_heads * head_dim
    if qkv.shape[1] != wq + 2 * wk or qkv.stride(1) != 1:
        raise ValueError("qkv must be [T, (Hq + 2 Hkv) * D] with contiguous rows")
    if positions.dtype != torch.int64 or positions.numel() != T or not positions.is_contiguous():
        raise ValueError("positions must be a contiguous int64 [T] tensor")
    if rope_table.dtype != torch.float32 or rope_table.shape[1] != head_dim or not rope_table.is_contiguous():
        raise ValueError("rope_table must be fp32 [positions, head_dim]")
    use_cache = k_cache is not None and k_cache.numel() > 0
    if use_cache and (slot_mapping is None or slot_mapping.dtype != torch.int64 or slot_mapping.numel() != T):
        raise ValueError("slot_mapping must be int64 [T]")
    q = torch.empty(T, num_q_heads, head_dim, dtype=qkv.dtype, device=qkv.device)
    k = torch.empty(T, num_kv_heads, head_dim, dtype=qkv.dtype, device=qkv.device)
    eps = VECTOR_NORM_EPS
    check(lib.b200_qk_norm_rope_store(
        qkv.data_ptr(), qkv.stride(0), q_norm_w.data_ptr(), k_norm_w.data_ptr(), rope_table.data_ptr(),
        rope_table.shape[0], positions.data_ptr(), q.data_ptr(), k.data_ptr(),
        k_cache.data_ptr() if use_cache else None, v_cache.data_ptr() if use_cache else None,
        slot_mapping.data_ptr() if use_cache else None, (k_cache.numel() // wk) if use_cache else 0, T,
        num_q_heads, num_kv_heads, head_dim, float(eps), _dt(qkv), status_word(dev).data_ptr(), _stream()),
        "qk_norm_rope_store")
    v = qkv[:, wq + wk:].view(T, num_kv_heads, head_dim)
    return q, k, v


def mla_prologue_supported(head_dim: int, rope_dim: int, kv_lora_rank: int, dtype: torch.dtype) -> bool:
    """Shapes the fused MLA pre-attention kernel takes (16-byte chunks everywhere, a rotation partner a whole
    number of lanes away); other shapes run the same stage as separate tensor operations on the device."""
    rpc = rope_dim // 8
    return (dtype == torch.bfloat16 and head_dim % 8 == 0 and rope_dim % 16 == 0 and kv_lora_rank % 8 == 0
            and rpc & (rpc - 1) == 0 and rpc <= 32)


def mla_prologue(q_up: torch.Tensor, kv_down: torch.Tensor, kv_norm_w: torch.Tensor, rope_table: torch.Tensor,
                 positions: torch.Tensor, num_heads: int, head_dim: int, rope_dim: int, kv_lora_rank: int,
                 latent_cache: torch.Tensor | None = None, slot_mapping: torch.Tensor | None = None):
    """MLA stage between the projections and the attention: q = [q_nope | RoPE(q_rope)] per head and the
    latent row [kv_norm(c) | RoPE(k_rope)], also scattered into the paged latent cache.

    q_up: [T, H*head_dim + H*rope_dim]; kv_down: [T, kv_lora_rank + rope_dim]; bf16.
    Returns (q [T, H, head_dim + rope_dim], rows [T, kv_lora_rank + rope_dim]).
    """
    dev = _cuda(q_up, kv_down, kv_norm_w, rope_table, positions, latent_cache, slot_mapping)
    T = q_up.shape[0]
    if q_up.dtype != torch.bfloat16 or kv_down.dtype != torch.bfloat16:
        raise ValueError("mla_prologue takes bf16 projections")
    if q_up.shape[1] != num_heads * (head_dim + rope_dim) or q_up.stride(1) != 1:
        raise ValueError("q_up must be [T, H*(head_dim + rope_dim)] with contiguous rows")
    if kv_down.shape != (T, kv_lora_rank + rope_dim) or kv_down.stride(1) != 1:
        raise ValueError("kv_down must be [T, kv_lora_rank + rope_dim] with contiguous rows")
    if positions.dtype != torch.int64 or positions.numel() != T or not positions.is_contiguous():
        raise ValueError("positions must be a contiguous int64 [T] tensor")
    if rope_table.dtype != torch.float32 or not rope_table.is_contiguous() or rope_table.dim() != 2:
        raise ValueError("rope_table must be a contiguous fp32 [positions, width] tensor")
    if kv_norm_w.dtype != torch.float32 or kv_norm_w.numel() != kv_lora_rank:
        raise ValueError("kv_norm_w must be fp32 [kv_lora_rank]")
    use_cache = latent_cache is not None and latent_cache.numel() > 0
    if use_cache:
        if latent_cache.dtype != torch.bfloat16 or latent_cache.shape[-1] != kv_lora_rank + rope_dim \
                or not latent_cache.is_contiguous():
            raise ValueError("latent_cache must be contiguous bf16 [..., kv_lora_rank + rope_dim]")
        if slot_mapping is None or slot_mapping.dtype != torch.int64 or slot_mapping.numel() != T:
            raise ValueError("slot_mapping must be int64 [T]")
    q = torch.empty(T, num_heads, head_dim + rope_dim, dtype=q_up.dtype, device=q_up.device)
    rows = torch.empty(T, kv_lora_rank + rope_dim, dtype=q_up.dtype, device=q_up.device)
    check(lib.b200_mla_prologue(
        q_up.data_ptr(), q_up.stride(0), kv_down.data_ptr(), kv_down.stride(0), kv_norm_w.data_ptr(),
        rope_table.data_ptr(), rope_table.shape[1], rope_table.shape[0], positions.data_ptr(), q.data_ptr(),
        rows.data_ptr(), latent_cache.data_ptr() if use_cache else None,
        slot_mapping.data_ptr() if use_cache else None,
        (latent_cache.numel() // (kv_lora_rank + rope_dim)) if use_cache else 0, T, num_heads, head_dim, rope_dim,
        kv_lora_rank, VECTOR_NORM_EPS, _dt(q_up), status_word(dev).data_ptr(), _stream()),
        "mla_prologue")
    return q, rows


MOE_ROUTE_MAX_EXPERTS, MOE_ROUTE_MAX_TOPK, MOE_ROUTE_MAX_TOKENS = 64, 8, 65536
MOE_GEMM_EARLY_LAUNCH = 0x100   # B200_MOE_GEMM_EARLY_LAUNCH


def moe_route(gate_logits: torch.Tensor, expert_bias: torch.Tensor, top_k: int, identity_tail: bool = False):
    """Top-k routing + grouping by expert.  Returns (sorted_token, sorted_expert, sorted_weight,
    expert_offsets, slot_to_row); see ``b200_moe_route`` in the header for the layout.  With
    ``identity_tail`` sorted_token has T more entries 0..T-1 at its end (rows of a shared expert)."""
    _cuda(gate_logits, expert_bias)
    T, E = gate_logits.shape
    if not gate_logits.is_contiguous() or expert_bias.dtype != torch.float32 or expert_bias.numel() != E:
        raise ValueError("gate_logits must be contiguous [T, E] and expert_bias fp32 [E]")
    dev, n = gate_logits.device, T * top_k
    tok = torch.empty(n + (T if identity_tail else 0), dtype=torch.int32, device=dev)
    exp = torch.empty(n, dtype=torch.int32, device=dev)
    w = torch.empty(n, dtype=gate_logits.dtype, device=dev)
    offs = torch.empty(E, dtype=torch.int32, device=dev)
    inv = torch.empty(T, top_k, dtype=torch.int32, device=dev)
    need = int(lib.b200_moe_route_workspace_bytes(T, E))
    ws = workspace(dev, need, "moe_route") if need else None
    check(lib.b200_moe_route(gate_logits.data_ptr(), expert_bias.data_ptr(), T, E, top_k, tok.data_ptr(),
                             exp.data_ptr(), w.data_ptr(), offs.data_ptr(), inv.data_ptr(), 1 if identity_tail else 0,
                             ws.data_ptr() if ws is not None else None, ws.numel() if ws is not None else 0,
                             _dt(gate_logits), _stream()), "moe_route")
    return tok, exp, w, offs, inv


MOE_GATE_ROUTE_MAX_TOKENS = 256
MOE_GATE_ROUTE_MAX_GATE_BYTES = 160 * 1024
MOE_GATE_ROUTE_GATHER_MAX_TOKENS = 32   # up to here the routing launch also copies the routed rows


def moe_gate_route(x: torch.Tensor, gate_w: torch.Tensor, expert_bias: torch.Tensor, top_k: int,
                   identity_tail: bool = False, gather: bool = False):
    """Gate projection + ``moe_route`` in one launch for at most 256 bf16 tokens.  Returns (sorted_token,
    sorted_expert, sorted_weight, expert_offsets, slot_to_row, gathered): ``gathered`` is x[sorted_token]
    when ``gather`` is set (meant for small batches: one thread block copies the rows), else None."""
    dev = _cuda(x, gate_w, expert_bias)
    T, d = x.shape
    E = gate_w.shape[0]
    if x.dtype != torch.bfloat16 or gate_w.dtype != torch.bfloat16 or not x.is_contiguous() \
            or not gate_w.is_contiguous() or gate_w.shape[1] != d:
        raise ValueError("x [T, d] and gate_w [E, d] must be contiguous bfloat16")
    if expert_bias.dtype != torch.float32 or expert_bias.numel() != E:
        raise ValueError("expert_bias must be fp32 [E]")
    n = T * top_k
    rows = n + (T if identity_tail else 0)
    tok = torch.empty(rows, dtype=torch.int32, device=dev)
    exp = torch.empty(n, dtype=torch.int32, device=dev)
    w = torch.empty(n, dtype=x.dtype, device=dev)
    offs = torch.empty(E, dtype=torch.int32, device=dev)
    inv = torch.empty(T, top_k, dtype=torch.int32, device=dev)
    xs = torch.empty(rows, d, dtype=x.dtype, device=dev) if gather else None
    ws = workspace(dev, int(lib.b200_moe_gate_route_workspace_bytes()), "moe_gate_route")
    check(lib.b200_moe_gate_route(x.data_ptr(), gate_w.data_ptr(), expert_bias.data_ptr(), T, E, top_k, d,
                                  tok.data_ptr(), exp.data_ptr(), w.data_ptr(), offs.data_ptr(), inv.data_ptr(),
                                  1 if identity_tail else 0, xs.data_ptr() if xs is not None else None,
                                  ws.data_ptr(), ws.numel(), _dt(x), _stream()), "moe_gate_route")
    return tok, exp, w, offs, inv, xs


def swiglu(h: torch.Tensor, bias: torch.Tensor | None = None, row_expert: torch.Tensor | None = None):
    """act = silu(h[:, :F] + b1) * (h[:, F:] + b3) for h [rows, 2F]; ``bias`` [experts, 2F] is indexed by
    ``row_expert`` [rows] int32 (row 0 without it); every intermediate is rounded to the dtype."""
    _cuda(h, bias, row_expert)
    rows, F2 = h.shape
    if not h.is_contiguous() or F2 % 2:
        raise ValueError("h must be contiguous [rows, 2*d_ff]")
    if bias is not None and (bias.dtype != h.dtype or not bias.is_contiguous() or bias.shape[-1] != F2):
        raise ValueError("bias must be contiguous [experts, 2*d_ff] in the dtype of h")
    if row_expert is not None and (row_expert.dtype != torch.int32 or row_expert.numel() != rows):
        raise ValueError("row_expert must be int32 [rows]")
    act = torch.empty(rows, F2 // 2, dtype=h.dtype, device=h.device)
    check(lib.b200_swiglu(h.data_ptr(), bias.data_ptr() if bias is not None else None,
                          row_expert.data_ptr() if row_expert is not None else None, act.data_ptr(), rows,
                          F2 // 2, _dt(h), _stream()), "swiglu")
    return act


def moe_grouped_gemm(x: torch.Tensor, w: torch.Tensor, expert_offsets: torch.Tensor,
                     bias: torch.Tensor | None = None, swiglu: bool = False, dense_rows: int = 0,
                     early_launch: bool = False) -> torch.Tensor:
    """Rows of x [R, k] grouped by expert (expert_offsets int32 [E], exclusive ends) times the expert's
    weight: w [E, n, k] -> [R, n]; with ``swiglu`` w is [E, 2*d_ff, k] = [w1 | w3], bias [E, 2*d_ff],
    and the result is silu(x w1^T + b1) * (x w3^T + b3) [R, d_ff].  bf16, tcgen05 tensor cores.
    ``dense_rows`` > 0: the last rows of x are not grouped and all use one more weight set, w[E] (w and
    bias then have E + 1 sets): a shared expert in the same launch."""
    _cuda(x, w, expert_offsets, bias)
    R, k = x.shape
    E, n, k2 = w.shape
    if dense_rows:
        E -= 1
    if x.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or not x.is_contiguous() or not w.is_contiguous():
        raise ValueError("x and w must be contiguous bfloat16")
    if k2 != k or expert_offsets.dtype != torch.int32 or expert_offsets.numel() != E or (swiglu and n % 2):
        raise ValueError("w must be [E, n, k] with k = x.shape[1]; expert_offsets int32 [E]")
    n_out = n // 2 if swiglu else n
    if bias is not None and (bias.dtype != torch.bfloat16 or not bias.is_contiguous()
                             or tuple(bias.shape) != (w.shape[0], n)):
        raise ValueError("bias must be contiguous bfloat16 [weight sets, n]")
    if dense_rows < 0 or dense_rows > R or E < 1:
        raise ValueError("dense_rows must be within the rows of x and leave at least one routed expert")
    out = torch.empty(R, n_out, dtype=torch.bfloat16, device=x.device)
    check(lib.b200_moe_grouped_gemm(x.data_ptr(), w.data_ptr(), bias.data_ptr() if bias is not None else None,
                                    out.data_ptr(), expert_offsets.data_ptr(), R, E, int(dense_rows), n_out, k,
                                    (1 if swiglu else 0) | (MOE_GEMM_EARLY_LAUNCH if early_launch else 0),
                                    _dt(x), status_word(x.device).data_ptr(), _stream()), "moe_grouped_gemm")
    return out


def lm_head_argmax_supported(hidden: torch.Tensor, w: torch.Tensor) -> bool:
    return (hidden.is_cuda and hidden.dtype == torch.bfloat16 and w.dtype == torch.bfloat16 and hidden.dim() == 2
            and hidden.shape[1] % 8 == 0 and hidden.shape[0] > 0)


def lm_head_argmax(hidden: torch.Tensor, w: torch.Tensor, bias: torch.Tensor | None = None,
                   out: torch.Tensor | None = None) -> torch.Tensor:
    """Greedy tokens of hidden [R, d] under the head w [vocab, d] (+ bias [vocab]): argmax over the bf16 logits,
    first maximum, without materialising the logits.  bf16; returns int64 [R]."""
    dev = _cuda(hidden, w, bias, out)
    R, d = hidden.shape
    V = w.shape[0]
    if hidden.dtype != torch.bfloat16 or w.dtype != torch.bfloat16 or not hidden.is_contiguous() \
            or not w.is_contiguous() or w.shape[1] != d:
        raise ValueError("hidden [R, d] and w [vocab, d] must be contiguous bfloat16")
    if bias is not None and (bias.dtype != torch.bfloat16 or bias.numel() != V or not bias.is_contiguous()):
        raise ValueError("bias must be contiguous bfloat16 [vocab]")
    if out is None:
        out = torch.empty(R, dtype=torch.int64, device=hidden.device)
    elif out.dtype != torch.int64 or out.numel() != R or not out.is_contiguous():
        raise ValueError("out must be a contiguous int64 [R] tensor")
    need = lib.b200_lm_head_argmax_workspace_bytes(R, V)
    ws = workspace(dev, need, "lm_head")
    check(lib.b200_lm_head_argmax(hidden.data_ptr(), w.data_ptr(), bias.data_ptr() if bias is not None else None,
                                  out.data_ptr(), R, V, d, ws.data_ptr(), ws.numel(), _dt(hidden),
                                  status_word(dev).data_ptr(), _stream()), "lm_head_argmax")
    return out


def moe_combine(expert_out: torch.Tensor, bias: torch.Tensor | None, row_expert: torch.Tensor,
                row_weight: torch.Tensor, slot_to_row: torch.Tensor, shared: torch.Tensor | None = None):
    """Weighted sum of every token's expert rows in ascending expert order (+ bias, + shared expert),
    rounding like the reference's accumulation in the activation dtype.  Returns [tokens, d]."""
    _cuda(expert_out, bias, row_expert, row_weight, slot_to_row, shared)
    T, K = slot_to_row.shape
    rows, d = expert_out.shape
    if rows != T * K or not expert_out.is_contiguous() or not slot_to_row.is_contiguous():
        raise ValueError("expert_out must be contiguous [tokens*top_k, d] and slot_to_row [tokens, top_k]")
    if row_weight.dtype != expert_out.dtype or row_weight.numel() != rows or row_expert.dtype != torch.int32:
        raise ValueError("row_weight must match expert_out's dtype, row_expert must be int32, both [rows]")
    if slot_to_row.dtype != torch.int32:
        raise ValueError("slot_to_row must be int32")
    for name, t, shape in (("bias", bias, None), ("shared", shared, (T, d))):
        if t is not None and (t.dtype != expert_out.dtype or not t.is_contiguous() or t.shape[-1] != d
                              or (shape is not None and tuple(t.shape) != shape)):
            raise ValueError(f"{name} must be contiguous [..., {d}] in the dtype of expert_out")
    out = torch.empty(T, d, dtype=expert_out.dtype, device=expert_out.device)
    check(lib.b200_moe_combine(expert_out.data_ptr(), bias.data_ptr() if bias is not None else None,
                               row_expert.data_ptr(), row_weight.data_ptr(), slot_to_row.data_ptr(),
                               shared.data_ptr() if shared is not None else None, out.data_ptr(), T, K, d,
                               _dt(expert_out), _stream()), "moe_combine")
    return out


def block_hash(token_ids, prefix: int = -1) -> int:
    """Chained XXH64 block hash; same value as BlockManager.compute_hash of the reference."""
    buf = array.array("i", token_ids)
    addr, n = buf.buffer_info()
    return int(lib.b200_block_hash(addr, n, 0 if prefix == -1 else prefix, 0 if prefix == -1 else 1))


def decode_advance(sampled: torch.Tensor, input_ids: torch.Tensor, context_lens: torch.Tensor,
                   slot_mapping: torch.Tensor, block_tables: torch.Tensor, block_size: int, num_blocks: int,
                   history: torch.Tensor | None = None) -> None:
    """Turns the decode inputs of the step that just sampled ``sampled`` into those of the next step, in
    place and on the device: input id = sampled token, context length + 1, slot of the new position from
    the block table (which must already list that block).  ``history`` [n] also receives the tokens."""
    dev = _cuda(sampled, input_ids, context_lens, slot_mapping, block_tables, history)
    n = sampled.numel()
    for t in (sampled, input_ids, context_lens, slot_mapping) + ((history,) if history is not None else ()):
        if t.dtype != torch.int64 or t.numel() < n or not t.is_contiguous():
            raise ValueError("sampled, input_ids, context_lens, slot_mapping, history must be contiguous int64 [n]")
    if block_tables.dtype != torch.int32 or block_tables.dim() != 2 or block_tables.shape[0] < n \
            or block_tables.stride(1) != 1:
        raise ValueError("block_tables must be int32 [n, max_blocks]")
    check(lib.b200_decode_advance(sampled.data_ptr(), input_ids.data_ptr(), context_lens.data_ptr(),
                                  slot_mapping.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
                                  int(block_size), int(num_blocks), n,
                                  history.data_ptr() if history is not None else None,
                                  status_word(dev).data_ptr(), _stream()), "decode_advance")


def block_table_patch(patches: torch.Tensor, count: int, block_tables: torch.Tensor) -> None:
    """Writes the first ``count`` (row, column, block id) int32 triples of ``patches`` into ``block_tables``
    [rows, max_blocks] on the device (incremental update of a device-resident table)."""
    if count <= 0:
        return
    dev = _cuda(patches, block_tables)
    if patches.dtype != torch.int32 or not patches.is_contiguous() or patches.numel() < 3 * count:
        raise ValueError("patches must be a contiguous int32 tensor of at least 3 * count elements")
    if block_tables.dtype != torch.int32 or block_tables.dim() != 2 or block_tables.stride(1) != 1:
        raise ValueError("block_tables must be int32 [rows, max_blocks]")
    check(lib.b200_block_table_patch(patches.data_ptr(), int(count), block_tables.data_ptr(), block_tables.stride(0),
                                     block_tables.shape[0], status_word(dev).data_ptr(), _stream()),
          "block_table_patch")


def block_hash_chain(token_ids, block_size: int) -> list[int]:
    """Chained XXH64 hashes of every full block of ``token_ids`` in one native call: element i is what
    ``block_hash(block i, prefix = element i-1)`` returns."""
    buf = array.array("i", token_ids)
    addr, n = buf.buffer_info()
    out = array.array("Q", bytes(8 * (n // block_size)))
    got = int(lib.b200_block_hash_chain(addr, n, block_size, out.buffer_info()[0]))
    if got != len(out):
        raise RuntimeError("b200_block_hash_chain failed")
    return out.tolist()


def sample(logits: torch.Tensor, temperatures: torch.Tensor | None, seed: int, offset: int,
           out: torch.Tensor | None = None) -> torch.Tensor:
    """One token per row of ``logits`` [B, V]: greedy where the temperature is <= 0 (or ``temperatures`` is
    None), else a draw from softmax(logits / T).  ``seed`` / ``offset`` select the random stream."""
    _cuda(logits, temperatures, out)
    B, V = logits.shape
    if logits.stride(1) != 1:
        raise ValueError("logits rows must be contiguous")
    if temperatures is not None and (temperatures.dtype != torch.float32 or temperatures.numel() != B
                                     or not temperatures.is_contiguous()):
        raise ValueError("temperatures must be contiguous float32 [B]")
    if out is None:
        out = torch.empty(B, dtype=torch.int64, device=logits.device)
    elif out.dtype != torch.int64 or out.numel() != B or not out.is_contiguous():
        raise ValueError("out must be contiguous int64 [B]")
    check(lib.b200_sample(logits.data_ptr(), logits.stride(0), temperatures.data_ptr() if temperatures is not None
                          else None, B, V, seed & 0xFFFFFFFFFFFFFFFF, offset & 0xFFFFFFFFFFFFFFFF, out.data_ptr(),
                          _dt(logits), _stream()), "sample")
    return out


# ------------------------------------------------------------------------------------------------
# residual streams, talking-heads attention, gated recurrence
# ------------------------------------------------------------------------------------------------
def _ptr(t: torch.Tensor | None):
    return t.data_ptr() if t is not None else None


def _f32vec(name: str, t: torch.Tensor | None, n: int) -> None:
    if t is not None and (t.dtype != torch.float32 or t.numel() != n or not t.is_contiguous()):
        raise ValueError(f"{name} must be a contiguous fp32 tensor of {n} elements")


def store_kv_rows(k: torch.Tensor, v: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                  slot_mapping: torch.Tensor) -> None:
    """``store_kvcache`` for pools whose key and value rows differ in width: k [T, Wk], v [T, Wv] (row stride
    free) into caches [num_blocks, block_size, heads, dim] with heads * dim == W; slots < 0 are skipped."""
    dev = _cuda(k, v, k_cache, v_cache, slot_mapping)
    T, wk = k.shape
    wv = v.shape[1]
    if v.shape[0] != T or k.stride(1) != 1 or v.stride(1) != 1:
        raise ValueError("k and v must be [T, width] with contiguous rows")
    if slot_mapping.dtype != torch.int64 or slot_mapping.numel() != T or not slot_mapping.is_contiguous():
        raise ValueError("slot_mapping must be a contiguous int64 tensor with one entry per token")
    slots = k_cache.shape[0] * k_cache.shape[1]
    if k_cache.numel() != slots * wk or v_cache.numel() != slots * wv or not k_cache.is_contiguous() \
            or not v_cache.is_contiguous() or any(t.dtype != k.dtype for t in (v, k_cache, v_cache)):
        raise ValueError("caches must be contiguous, of k's dtype, with the same slots and rows as wide as k / v")
    check(lib.b200_store_kv_rows(k.data_ptr(), v.data_ptr(), k.stride(0), v.stride(0), k_cache.data_ptr(),
                                 v_cache.data_ptr(), slot_mapping.data_ptr(), T, wk, wv, slots, _dt(k),
                                 status_word(dev).data_ptr(), _stream()), "store_kv_rows")


def stream_update(x: torch.Tensor, norm_w: torch.Tensor, eps: float, dtype: torch.dtype, *,
                  tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None,
                  y: torch.Tensor | None = None, y1: torch.Tensor | None = None,
                  join_w: tuple[torch.Tensor, torch.Tensor] | None = None, join_eps: float = 0.0,
                  layer_scale: torch.Tensor | None = None, mix: torch.Tensor | None = None,
                  out_w: torch.Tensor | None = None, in_w: torch.Tensor | None = None, plus_one: bool = True):
    """One sublayer boundary of a decoder with fp32 residual streams x [T, S, d], in place
    (``b200_stream_update``): write the sublayer result ``y`` (or the join of ``y`` and ``y1``) back into the
    streams, read the next sublayer's input from them and return its norm [T, d] in ``dtype``.  With
    ``embed`` / ``tokens`` the streams start from the embedding rows instead of an update."""
    dev = _cuda(x, norm_w, tokens, embed, y, y1, layer_scale, mix, out_w, in_w)
    T, S, d = x.shape
    if x.dtype != torch.float32 or not x.is_contiguous():
        raise ValueError("x must be a contiguous fp32 [T, streams, d] tensor")
    for name, t, n in (("norm_w", norm_w, d), ("layer_scale", layer_scale, d), ("mix", mix, S * S), ("out_w", out_w, S),
                       ("in_w", in_w, S)) + ((("join_w", join_w[0], d), ("join_w", join_w[1], d)) if join_w else ()):
        _f32vec(name, t, n)
    for t in (y, y1):
        if t is not None and (t.shape != (T, d) or t.dtype != dtype or not t.is_contiguous()):
            raise ValueError("y must be contiguous [T, d] in the activation dtype")
    if embed is not None and (embed.shape[1] != d or embed.dtype != dtype or not embed.is_contiguous()
                              or tokens is None or tokens.dtype != torch.int64 or tokens.numel() != T):
        raise ValueError("embed must be contiguous [vocab, d] in the activation dtype, tokens int64 [T]")
    h = torch.empty(T, d, dtype=dtype, device=x.device)
    check(lib.b200_stream_update(
        x.data_ptr(), _ptr(tokens) if embed is not None else None, _ptr(embed), embed.shape[0] if embed is not None else 0,
        _ptr(y), _ptr(y1), _ptr(join_w[0]) if join_w else None, _ptr(join_w[1]) if join_w else None, float(join_eps),
        _ptr(layer_scale), _ptr(mix), _ptr(out_w), _ptr(in_w), norm_w.data_ptr(), 1 if plus_one else 0, float(eps),
        h.data_ptr(), T, S, d, _dt(h), status_word(dev).data_ptr(), _stream()), "stream_update")
    return h


def clamped_glu(h: torch.Tensor, limit: float, slope: float) -> torch.Tensor:
    """g sigmoid(slope g) (u + 1) for h = [gate | up] [rows, 2F], g = min(gate, limit), u = clamp(up, +-limit)."""
    _cuda(h)
    rows, F2 = h.shape
    if not h.is_contiguous() or F2 % 2:
        raise ValueError("h must be contiguous [rows, 2*d_ff]")
    act = torch.empty(rows, F2 // 2, dtype=h.dtype, device=h.device)
    check(lib.b200_clamped_glu(h.data_ptr(), act.data_ptr(), rows, F2 // 2, float(limit), float(slope), _dt(h),
                               _stream()), "clamped_glu")
    return act


TALKING_TILE_ROWS = 16              # B200_TALKING_TILE_ROWS


class TalkingHeads:
    """Constants of a talking-heads attention layer on the device: the score scale and cap, the distance bias
    (r1, r2 [H]), the head mix ``talk`` [H, H] (out, in) and the window (0: none).  The bias of every distance
    inside the window is tabulated once."""

    max_table = 1 << 16

    def __init__(self, scale: float, softcap: float, r1: torch.Tensor, r2: torch.Tensor, talk: torch.Tensor, window: int,
                 device):
        H = talk.shape[0]
        self.scale, self.softcap, self.window, self.H = float(scale), float(softcap), int(window), H
        host = talk.detach().float().cpu().contiguous()
        self.talk = host.to(device)
        self.r1 = r1.detach().float().to(device).contiguous()
        self.r2 = r2.detach().float().to(device).contiguous()
        for name, t, n in (("r1", self.r1, H), ("r2", self.r2, H), ("talk", self.talk, H * H)):
            _f32vec(name, t, n)
        self.consts_host = torch.cat([host.reshape(-1), r1.detach().float().cpu(), r2.detach().float().cpu()]).contiguous()
        self.table = None
        if 0 < self.window <= self.max_table:
            dist = torch.arange(self.window, dtype=torch.float64)[None, :]
            t = r1.detach().double().cpu()[:, None] * torch.log1p(r2.detach().double().cpu()[:, None] * dist)
            self.table = t.float().to(device).contiguous()       # [H, window]


def talking_attention(q: torch.Tensor, gate: torch.Tensor | None, k_cache: torch.Tensor, v_cache: torch.Tensor,
                      block_tables: torch.Tensor, c: TalkingHeads, *, cu_seqlens_q: torch.Tensor | None = None,
                      cu_seqlens_k: torch.Tensor | None = None, context_lens: torch.Tensor | None = None,
                      max_seqlen_q: int = 1, plan: "PrefillPlan | None" = None, out: torch.Tensor | None = None,
                      general: bool = False) -> torch.Tensor:
    """Attention of ``b200_talking_attention`` over the paged pool: q [rows, H * dk], gate [rows, H * dv] (row
    strides free), caches [num_blocks, block_size, Hkv, d*].  Rows are ragged (``cu_seqlens_*``) or one per sequence
    (``context_lens``); ``plan``: tile list of the step for ``TALKING_TILE_ROWS`` rows.  ``general`` forces the general kernel.  Returns [rows, H, dv]."""
    dev = _cuda(q, gate, k_cache, v_cache, block_tables, cu_seqlens_q, cu_seqlens_k, context_lens, out)
    rows, H = q.shape[0], c.H
    nb, bs, Hkv, dk = k_cache.shape
    dv = v_cache.shape[3]
    if v_cache.shape[:3] != (nb, bs, Hkv) or not k_cache.is_contiguous() or not v_cache.is_contiguous() \
            or k_cache.dtype != q.dtype or v_cache.dtype != q.dtype:
        raise ValueError("caches must be contiguous [num_blocks, block_size, Hkv, d] of q's dtype")
    if q.shape[1] != H * dk or q.stride(1) != 1 or (gate is not None and (gate.shape != (rows, H * dv)
                                                    or gate.stride(1) != 1 or gate.dtype != q.dtype)):
        raise ValueError("q must be [rows, H * dk] and gate [rows, H * dv] with contiguous rows")
    if cu_seqlens_q is not None:
        n = cu_seqlens_q.numel() - 1
        if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k is None or cu_seqlens_k.dtype != torch.int32 \
                or cu_seqlens_k.numel() != n + 1:
            raise ValueError("cu_seqlens must be int32 tensors of the same length")
    else:
        n = rows
        if context_lens is None or context_lens.dtype != torch.int64 or context_lens.numel() < rows:
            raise ValueError("context_lens must be int64 with one entry per row")
    if block_tables.dtype != torch.int32 or block_tables.shape[0] < n or block_tables.stride(1) != 1:
        raise ValueError("block_tables must be int32 [num_seqs, max_blocks]")
    if out is None:
        out = torch.empty(rows, H, dv, dtype=q.dtype, device=q.device)
    elif out.shape != (rows, H, dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [rows, H, dv] tensor")
    need = int(lib.b200_talking_attention_workspace_bytes(n, H, dv, c.window, 0 if cu_seqlens_q is not None else 1, _dt(q)))
    ws = workspace(dev, need, "talking") if need else None
    check(lib.b200_talking_attention(
        q.data_ptr(), q.stride(0), _ptr(gate), gate.stride(0) if gate is not None else 0, k_cache.data_ptr(),
        v_cache.data_ptr(), out.data_ptr(), block_tables.data_ptr(), block_tables.stride(0), bs, nb, _ptr(cu_seqlens_q),
        _ptr(cu_seqlens_k), _ptr(context_lens), n, rows, int(max_seqlen_q), H, Hkv, dk, dv, c.scale, c.softcap,
        c.r1.data_ptr(), c.r2.data_ptr(), c.talk.data_ptr(), None if general else c.consts_host.data_ptr(), _ptr(c.table),
        c.table.shape[1] if c.table is not None else 0, c.window,
        plan.buffer.data_ptr() if plan is not None else None, plan.tile_rows if plan is not None else 0,
        plan.capacity if plan is not None else 0, _ptr(ws), ws.numel() if ws is not None else 0, _dt(q),
        status_word(dev).data_ptr(), _stream()), "talking_attention")
    return out


def gated_recurrence(q: torch.Tensor, f: torch.Tensor, v: torch.Tensor, f_bias: torch.Tensor, lower: torch.Tensor,
                     norm_w: torch.Tensor, eps: float, state: torch.Tensor, state_slots: torch.Tensor, *,
                     cu_seqlens_q: torch.Tensor | None = None, cu_seqlens_k: torch.Tensor | None = None,
                     context_lens: torch.Tensor | None = None, max_seqlen_q: int = 1) -> torch.Tensor:
    """Gated linear recurrence of ``b200_gated_recurrence``: q, f [T, heads * dk], v [T, heads * dv] (views of one
    projection), state fp32 [slots, heads, dk, dv] updated in place.  Returns the normed heads [T, heads * dv]."""
    dev = _cuda(q, f, v, f_bias, lower, norm_w, state, state_slots, cu_seqlens_q, cu_seqlens_k, context_lens)
    slots, H, dk, dv = state.shape
    T = q.shape[0]
    if q.shape != (T, H * dk) or f.shape != (T, H * dk) or v.shape != (T, H * dv) or any(
            t.stride(1) != 1 or t.stride(0) != q.stride(0) or t.dtype != q.dtype for t in (q, f, v)):
        raise ValueError("q, f [T, H * dk] and v [T, H * dv] must share dtype and row stride")
    if state.dtype != torch.float32 or not state.is_contiguous():
        raise ValueError("state must be contiguous fp32 [slots, H, dk, dv]")
    for name, t, n in (("f_bias", f_bias, H * dk), ("lower", lower, H * dk), ("norm_w", norm_w, dv)):
        _f32vec(name, t, n)
    n = cu_seqlens_q.numel() - 1 if cu_seqlens_q is not None else T
    if state_slots.dtype != torch.int64 or state_slots.numel() < n or not state_slots.is_contiguous():
        raise ValueError("state_slots must be contiguous int64 with one entry per sequence")
    if cu_seqlens_q is not None:
        if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k is None or cu_seqlens_k.dtype != torch.int32:
            raise ValueError("cu_seqlens must be int32")
    elif context_lens is None or context_lens.dtype != torch.int64 or context_lens.numel() < n:
        raise ValueError("context_lens must be int64 with one entry per row")
    out = torch.empty(T, H * dv, dtype=q.dtype, device=q.device)
    need = int(lib.b200_gated_recurrence_workspace_bytes(n, T, int(max_seqlen_q), H, dk, dv))
    ws = workspace(dev, need, "recurrence") if need else None
    check(lib.b200_gated_recurrence(
        q.data_ptr(), f.data_ptr(), v.data_ptr(), q.stride(0), f_bias.data_ptr(), lower.data_ptr(), norm_w.data_ptr(),
        float(eps), state.data_ptr(), slots, state_slots.data_ptr(), _ptr(cu_seqlens_q), _ptr(cu_seqlens_k),
        _ptr(context_lens), n, T, int(max_seqlen_q), H, dk, dv, out.data_ptr(), _ptr(ws),
        ws.numel() if ws is not None else 0, _dt(q), status_word(dev).data_ptr(), _stream()), "gated_recurrence")
    return out


# ------------------------------------------------------------------------------------------------
# post-norm residual, per-head norms with interleaved rotation, latent rows, gated delta rule
# ------------------------------------------------------------------------------------------------
def residual_norm(x: torch.Tensor, eps: float, dtype: torch.dtype, *, tokens: torch.Tensor | None = None,
                  embed: torch.Tensor | None = None, y: torch.Tensor | None = None, norm_w: torch.Tensor | None = None,
                  final_w: torch.Tensor | None = None) -> torch.Tensor:
    """One sublayer boundary with a norm on the sublayer's output (``b200_residual_norm``): x [T, d] fp32 takes the normed
    ``y`` (or starts as the rows ``tokens`` of ``embed``) in place; returns x, or its norm with ``final_w``, in ``dtype``."""
    dev = _cuda(x, tokens, embed, y, norm_w, final_w)
    T, d = x.shape
    if x.dtype != torch.float32 or not x.is_contiguous():
        raise ValueError("x must be a contiguous fp32 [T, d] tensor")
    _f32vec("norm_w", norm_w, d)
    _f32vec("final_w", final_w, d)
    if embed is not None:
        if embed.shape[1] != d or embed.dtype != dtype or not embed.is_contiguous() or tokens is None \
                or tokens.dtype != torch.int64 or tokens.numel() != T:
            raise ValueError("embed must be contiguous [vocab, d] in the activation dtype, tokens int64 [T]")
    elif y is None or norm_w is None or y.shape != (T, d) or y.dtype != dtype or not y.is_contiguous():
        raise ValueError("y must be contiguous [T, d] in the activation dtype, with its norm weight")
    h = torch.empty(T, d, dtype=dtype, device=x.device)
    check(lib.b200_residual_norm(x.data_ptr(), _ptr(tokens) if embed is not None else None, _ptr(embed),
                                 embed.shape[0] if embed is not None else 0, _ptr(y), _ptr(norm_w), _ptr(final_w), float(eps),
                                 h.data_ptr(), T, d, _dt(h), status_word(dev).data_ptr(), _stream()), "residual_norm")
    return h


@dataclass(frozen=True)
class YarnScaling:
    """YaRN stretching of rotary frequencies: pairs that turn fewer than ``slow`` times within ``original`` positions turn
    ``factor`` times slower, those that turn more than ``fast`` times as they are, those between on a linear ramp."""
    factor: float
    original: float
    fast: float
    slow: float

    @property
    def magnitude(self) -> float:
        """What cos and sin are multiplied by."""
        return 0.1 * math.log(self.factor) + 1.0

    def pair(self, turns: float, base: float, dims: int) -> float:
        """Index (real) of the pair that turns ``turns`` times within ``original`` positions."""
        return dims * math.log(self.original / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    def ramp(self, base: float, dims: int) -> torch.Tensor:
        """How far every pair is stretched, 0 to 1."""
        first = max(math.floor(self.pair(self.fast, base, dims)), 0)
        last = min(math.ceil(self.pair(self.slow, base, dims)), dims - 1)
        i = torch.arange(dims // 2, dtype=torch.float64)
        return ((i - first) / max(last - first, 0.001)).clamp(0.0, 1.0)


def rotary_frequencies(base: float, dims: int, device, scaling: YarnScaling | None = None) -> torch.Tensor:
    """base^(-2i / dims), i < dims / 2, in fp64, stretched by ``scaling``."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    freq = float(base) ** (-2.0 * i / max(dims, 1))
    if scaling is not None and dims:
        ramp = scaling.ramp(float(base), dims)
        freq = freq / scaling.factor * ramp + freq * (1.0 - ramp)
    return freq.to(device)


def head_norm_rope_store(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, q_norm_w: torch.Tensor, k_norm_w: torch.Tensor,
                         eps: float, freq: torch.Tensor, positions: torch.Tensor, k_cache: torch.Tensor,
                         v_cache: torch.Tensor, slot_mapping: torch.Tensor):
    """Norm of every query / key head, interleaved rotation of its first 2 * freq.numel() channels, scatter of k and v
    (``b200_head_norm_rope_store``).  q [T, Hq * D], k [T, Hkv * D], v [T, Hkv * Dv] are views of one projection; caches
    [num_blocks, block_size, Hkv, D*].  Returns (q [T, Hq, D], k [T, Hkv, D])."""
    dev = _cuda(q, k, v, q_norm_w, k_norm_w, freq, positions, k_cache, v_cache, slot_mapping)
    T, D = q.shape[0], q_norm_w.numel()
    nb, bs, Hkv, Dc = k_cache.shape
    Dv, Hq = v_cache.shape[3], q.shape[1] // D
    if Dc != D or v_cache.shape[:3] != (nb, bs, Hkv) or not k_cache.is_contiguous() or not v_cache.is_contiguous() \
            or k_cache.dtype != q.dtype or v_cache.dtype != q.dtype:
        raise ValueError("caches must be contiguous [num_blocks, block_size, Hkv, d] of q's dtype")
    if q.shape != (T, Hq * D) or k.shape != (T, Hkv * D) or v.shape != (T, Hkv * Dv) or any(
            t.stride(1) != 1 or t.stride(0) != q.stride(0) or t.dtype != q.dtype for t in (q, k, v)):
        raise ValueError("q, k, v must share dtype and row stride")
    _f32vec("q_norm_w", q_norm_w, D)
    _f32vec("k_norm_w", k_norm_w, D)
    if freq.dtype != torch.float64 or not freq.is_contiguous():
        raise ValueError("freq must be contiguous fp64")
    for name, t in (("positions", positions), ("slot_mapping", slot_mapping)):
        if t.dtype != torch.int64 or t.numel() != T or not t.is_contiguous():
            raise ValueError(f"{name} must be contiguous int64 with one entry per token")
    qo = torch.empty(T, Hq, D, dtype=q.dtype, device=q.device)
    ko = torch.empty(T, Hkv, D, dtype=q.dtype, device=q.device)
    check(lib.b200_head_norm_rope_store(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), q.stride(0), q_norm_w.data_ptr(), k_norm_w.data_ptr(), float(eps),
        freq.data_ptr(), 2 * freq.numel(), positions.data_ptr(), qo.data_ptr(), ko.data_ptr(), k_cache.data_ptr(),
        v_cache.data_ptr(), slot_mapping.data_ptr(), nb * bs, T, Hq, Hkv, D, Dv, _dt(q), status_word(dev).data_ptr(),
        _stream()), "head_norm_rope_store")
    return qo, ko


def latent_norm_store(rows: torch.Tensor, norm_w: torch.Tensor, eps: float, cache: torch.Tensor,
                      slot_mapping: torch.Tensor) -> torch.Tensor:
    """RMS norm of latent rows [T, r] (row stride free), written to cache[slot_mapping] and returned [T, r]."""
    dev = _cuda(rows, norm_w, cache, slot_mapping)
    T, r = rows.shape
    _f32vec("norm_w", norm_w, r)
    if rows.stride(1) != 1 or cache.shape[-1] != r or cache.dtype != rows.dtype or not cache.is_contiguous():
        raise ValueError("rows/cache shape, dtype or layout mismatch")
    if slot_mapping.dtype != torch.int64 or slot_mapping.numel() != T or not slot_mapping.is_contiguous():
        raise ValueError("slot_mapping must be a contiguous int64 tensor with one entry per row")
    out = torch.empty(T, r, dtype=rows.dtype, device=rows.device)
    check(lib.b200_latent_norm_store(rows.data_ptr(), rows.stride(0), norm_w.data_ptr(), float(eps), out.data_ptr(),
                                     cache.data_ptr(), slot_mapping.data_ptr(), cache.numel() // r, T, r, _dt(rows),
                                     status_word(dev).data_ptr(), _stream()), "latent_norm_store")
    return out


def gather_rows(cache: torch.Tensor, block_tables: torch.Tensor, cu_seqlens_k: torch.Tensor, max_seqlen_k: int,
                total: int, cu_seqlens_full: torch.Tensor | None = None, multiple: int = 1) -> torch.Tensor:
    """Rows of whole contexts, packed [total, W], from a pool [num_blocks, block_size, W] through the block tables.  With
    ``cu_seqlens_full`` (the contexts' own offsets) ``cu_seqlens_k`` counts the last rows of every context.  ``multiple``:
    the result is padded with zero rows to a multiple of this many."""
    dev = _cuda(cache, block_tables, cu_seqlens_k, cu_seqlens_full)
    nb, bs, W = cache.shape
    n = cu_seqlens_k.numel() - 1
    if not cache.is_contiguous() or block_tables.dtype != torch.int32 or block_tables.shape[0] < n \
            or block_tables.stride(1) != 1 or cu_seqlens_k.dtype != torch.int32:
        raise ValueError("cache must be contiguous, block_tables int32 [n, max_blocks], cu_seqlens_k int32 [n + 1]")
    total = -(-total // multiple) * multiple
    out = torch.empty(total, W, dtype=cache.dtype, device=cache.device)
    if cu_seqlens_full is not None and (cu_seqlens_full.dtype != torch.int32 or cu_seqlens_full.numel() != n + 1):
        raise ValueError("cu_seqlens_full must be int32 [n + 1]")
    check(lib.b200_gather_last_rows(cache.data_ptr(), bs, nb, W * cache.element_size(), block_tables.data_ptr(),
                                    block_tables.stride(0), cu_seqlens_k.data_ptr(), _ptr(cu_seqlens_full), n,
                                    int(max_seqlen_k), out.data_ptr(), total, status_word(dev).data_ptr(), _stream()),
          "gather_rows")
    return out


def sigmoid_gate(o: torch.Tensor, gate: torch.Tensor) -> torch.Tensor:
    """o * sigmoid(gate) in place; o contiguous [T, W], gate [T, W] with a free row stride."""
    _cuda(o, gate)
    if o.shape != gate.shape or not o.is_contiguous() or gate.stride(1) != 1 or gate.dtype != o.dtype:
        raise ValueError("o must be contiguous [T, W] and gate [T, W] of its dtype with contiguous rows")
    check(lib.b200_sigmoid_gate(o.data_ptr(), gate.data_ptr(), gate.stride(0), o.shape[0], o.shape[1], _dt(o), _stream()),
          "sigmoid_gate")
    return o


def squared_relu(x: torch.Tensor) -> torch.Tensor:
    """max(x, 0)^2 in place."""
    _cuda(x)
    if not x.is_contiguous():
        raise ValueError("x must be contiguous")
    check(lib.b200_squared_relu(x.data_ptr(), x.numel(), _dt(x), _stream()), "squared_relu")
    return x


def softcap_logits(logits: torch.Tensor, scale: float, cap: float) -> torch.Tensor:
    """cap * tanh(scale * logits / cap) in place on fp32 logits (cap <= 0: scale only)."""
    _cuda(logits)
    if logits.dtype != torch.float32 or not logits.is_contiguous():
        raise ValueError("logits must be contiguous fp32")
    check(lib.b200_softcap_logits(logits.data_ptr(), logits.numel(), float(scale), float(cap), _stream()), "softcap_logits")
    return logits


class DeltaRule:
    """Constants of a gated delta rule layer on the device: head layout, convolution weights over the projection columns
    [q | k | v] (``columns``: first column of each; ``width``: columns in all, weights [taps, width]), gate biases, norm."""

    def __init__(self, heads: int, kv_heads: int, dim: int, vdim: int, columns: tuple[int, int, int], conv_w: torch.Tensor,
                 dt_bias: torch.Tensor, a_log: torch.Tensor, norm_w: torch.Tensor, eps: float):
        self.heads, self.kv_heads, self.dim, self.vdim, self.columns, self.eps = heads, kv_heads, dim, vdim, columns, float(eps)
        self.taps, self.width = conv_w.shape
        self.conv_w, self.dt_bias, self.a_log, self.norm_w = conv_w, dt_bias, a_log, norm_w
        for name, t, n in (("conv_w", conv_w, self.taps * self.width), ("dt_bias", dt_bias, heads), ("a_log", a_log, heads),
                           ("norm_w", norm_w, vdim)):
            _f32vec(name, t, n)


def _delta_inputs(c: DeltaRule, proj: torch.Tensor, b, a, gate, state: torch.Tensor, ring: torch.Tensor,
                  state_slots: torch.Tensor, n: int) -> None:
    T = proj.shape[0]
    H, dk, dv = c.heads, c.dim, c.vdim
    if proj.shape[1] < c.width or proj.stride(1) != 1 or b.shape != (T, H) or a.shape != (T, H) or gate.shape != (T, H * dv) \
            or any(t.stride(1) != 1 or t.stride(0) != proj.stride(0) or t.dtype != proj.dtype for t in (b, a, gate)):
        raise ValueError("proj [T, >= width], b and a [T, heads], gate [T, heads * vdim] must share dtype and row stride")
    slots = state.shape[0]
    if state.dtype != torch.float32 or state.shape != (slots, H, dk, dv) or not state.is_contiguous() \
            or ring.dtype != torch.float32 or ring.shape != (slots, c.taps, c.width) or not ring.is_contiguous():
        raise ValueError("state must be fp32 [slots, heads, dim, vdim] and the ring fp32 [slots, taps, width]")
    if state_slots.dtype != torch.int64 or state_slots.numel() < n or not state_slots.is_contiguous():
        raise ValueError("state_slots must be contiguous int64 with one entry per sequence")


def delta_rule(c: DeltaRule, proj: torch.Tensor, b: torch.Tensor, a: torch.Tensor, gate: torch.Tensor, state: torch.Tensor,
               ring: torch.Tensor, state_slots: torch.Tensor, cu_seqlens_q: torch.Tensor, cu_seqlens_k: torch.Tensor,
               out: torch.Tensor | None = None, general: bool = False) -> torch.Tensor:
    """Gated delta rule of ragged portions (``b200_delta_conv`` and ``b200_delta_rule``): proj [T, >= width] with the raw
    [q | k | v] columns, b, a, gate views with the same row stride; state and convolution ring advance in place.
    ``general`` forces the token-by-token kernel.  Returns the gated heads [T, heads * vdim]."""
    dev = _cuda(proj, b, a, gate, state, ring, state_slots, cu_seqlens_q, cu_seqlens_k, out)
    T, n = proj.shape[0], cu_seqlens_q.numel() - 1
    _delta_inputs(c, proj, b, a, gate, state, ring, state_slots, n)
    if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k.dtype != torch.int32 or cu_seqlens_k.numel() != n + 1:
        raise ValueError("cu_seqlens must be int32 tensors of the same length")
    out = _delta_out(c, proj, out)
    act = torch.empty(T, c.width, dtype=proj.dtype, device=proj.device)
    check(lib.b200_delta_conv(proj.data_ptr(), proj.stride(0), c.conv_w.data_ptr(), c.taps, c.width, ring.data_ptr(),
                              ring.shape[0], state_slots.data_ptr(), cu_seqlens_q.data_ptr(), cu_seqlens_k.data_ptr(), n, T,
                              act.data_ptr(), _dt(proj), status_word(dev).data_ptr(), _stream()), "delta_conv")
    need = 0 if general else int(lib.b200_delta_rule_workspace_bytes(n, T, c.heads, c.dim, c.vdim, _dt(proj)))
    ws = workspace(dev, need, "delta") if need else None
    q, k, v = (act[:, at:] for at in c.columns)
    check(lib.b200_delta_rule(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), act.stride(0), b.data_ptr(), a.data_ptr(), gate.data_ptr(), proj.stride(0),
        c.dt_bias.data_ptr(), c.a_log.data_ptr(), c.norm_w.data_ptr(), c.eps, state.data_ptr(), state.shape[0],
        state_slots.data_ptr(), cu_seqlens_q.data_ptr(), cu_seqlens_k.data_ptr(), n, T, c.heads, c.kv_heads, c.dim, c.vdim,
        out.data_ptr(), _ptr(ws), ws.numel() if ws is not None else 0, _dt(proj), status_word(dev).data_ptr(), _stream()),
        "delta_rule")
    return out


def delta_step(c: DeltaRule, proj: torch.Tensor, b: torch.Tensor, a: torch.Tensor, gate: torch.Tensor, state: torch.Tensor,
               ring: torch.Tensor, state_slots: torch.Tensor, context_lens: torch.Tensor,
               out: torch.Tensor | None = None) -> torch.Tensor:
    """One token per sequence of the gated delta rule, convolution included (``b200_delta_step``); row i of the inputs is
    sequence i, ``context_lens[i]`` tokens long with it.  Rows beyond ``context_lens`` are left alone."""
    dev = _cuda(proj, b, a, gate, state, ring, state_slots, context_lens, out)
    n = context_lens.numel()
    _delta_inputs(c, proj, b, a, gate, state, ring, state_slots, n)
    if context_lens.dtype != torch.int64 or n > proj.shape[0] or not context_lens.is_contiguous():
        raise ValueError("context_lens must be contiguous int64 with at most one entry per row")
    out = _delta_out(c, proj, out)
    q, k, v = (proj[:, at:] for at in c.columns)
    check(lib.b200_delta_step(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), b.data_ptr(), a.data_ptr(), gate.data_ptr(), proj.stride(0),
        c.conv_w.data_ptr(), c.taps, c.width, *c.columns, ring.data_ptr(), c.dt_bias.data_ptr(), c.a_log.data_ptr(),
        c.norm_w.data_ptr(), c.eps, state.data_ptr(), state.shape[0], state_slots.data_ptr(), context_lens.data_ptr(), n,
        c.heads, c.kv_heads, c.dim, c.vdim, out.data_ptr(), _dt(proj), status_word(dev).data_ptr(), _stream()), "delta_step")
    return out


def _delta_out(c: DeltaRule, proj: torch.Tensor, out: torch.Tensor | None) -> torch.Tensor:
    shape = (proj.shape[0], c.heads * c.vdim)
    if out is None:
        return torch.empty(shape, dtype=proj.dtype, device=proj.device)
    if out.shape != shape or out.dtype != proj.dtype or not out.is_contiguous():
        raise ValueError("out must be contiguous [T, heads * vdim] of proj's dtype")
    return out


# ------------------------------------------------------------------------------------------------
# parallel gated sublayers, windowed latent attention, grouped expert routing, token inputs
# ------------------------------------------------------------------------------------------------
def _tokens(name: str, t: torch.Tensor, n: int) -> None:
    if t.dtype != torch.int64 or t.numel() != n or not t.is_contiguous():
        raise ValueError(f"{name} must be contiguous int64 with one entry per token")


def residual_group_norm(x: torch.Tensor, norm_w: torch.Tensor, groups: int, eps: float, dtype: torch.dtype, *,
                        y: torch.Tensor | None = None, y_norm_w: torch.Tensor | None = None,
                        tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, embed_scale: float = 1.0,
                        start: bool = False) -> torch.Tensor:
    """One layer boundary (``b200_residual_group_norm``): x [T, d] fp32 takes the normed ``y`` and the scaled embedding rows
    (either may be absent; ``start``: x begins as zero) in place; returns its norm in ``groups`` parts, in ``dtype``."""
    dev = _cuda(x, norm_w, y, y_norm_w, tokens, embed)
    T, d = x.shape
    if x.dtype != torch.float32 or not x.is_contiguous():
        raise ValueError("x must be a contiguous fp32 [T, d] tensor")
    _f32vec("norm_w", norm_w, d)
    _f32vec("y_norm_w", y_norm_w, d)
    if y is not None and (y_norm_w is None or y.shape != (T, d) or y.dtype != dtype or not y.is_contiguous()):
        raise ValueError("y must be contiguous [T, d] in the activation dtype, with its norm weight")
    if embed is not None:
        if embed.shape[1] != d or embed.dtype != dtype or not embed.is_contiguous() or tokens is None:
            raise ValueError("embed must be contiguous [vocab, d] in the activation dtype, with tokens")
        _tokens("tokens", tokens, T)
    h = torch.empty(T, d, dtype=dtype, device=x.device)
    check(lib.b200_residual_group_norm(
        x.data_ptr(), _ptr(y), _ptr(y_norm_w), _ptr(tokens) if embed is not None else None, _ptr(embed),
        embed.shape[0] if embed is not None else 0, float(embed_scale), 1 if start else 0, norm_w.data_ptr(), int(groups),
        float(eps), h.data_ptr(), T, d, _dt(h), status_word(dev).data_ptr(), _stream()), "residual_group_norm")
    return h


def gated_residual(x: torch.Tensor, y1: torch.Tensor, gate1: torch.Tensor, y2: torch.Tensor | None = None,
                   gate2: torch.Tensor | None = None, row_weight: torch.Tensor | None = None,
                   slot_to_row: torch.Tensor | None = None) -> torch.Tensor:
    """x [T, d] fp32 <- x + y1 sigmoid(gate1) + y2 sigmoid(gate2) in place; gates [T, d] are views of one projection.  With
    ``row_weight`` / ``slot_to_row`` [T, top] y2 holds expert rows [T * top, d].  Returns x in the dtype of y1."""
    dev = _cuda(x, y1, gate1, y2, gate2, row_weight, slot_to_row)
    T, d = x.shape
    top = slot_to_row.shape[1] if slot_to_row is not None else 0
    if x.dtype != torch.float32 or not x.is_contiguous() or y1.shape != (T, d) or not y1.is_contiguous():
        raise ValueError("x must be contiguous fp32 [T, d], y1 contiguous [T, d]")
    for g in (gate1, gate2):
        if g is not None and (g.shape != (T, d) or g.dtype != y1.dtype or g.stride(1) != 1 or g.stride(0) != gate1.stride(0)):
            raise ValueError("gates must be [T, d] in the dtype of y1 with one row stride")
    if y2 is not None and (gate2 is None or y2.shape != ((T * top) if top else T, d) or y2.dtype != y1.dtype
                           or not y2.is_contiguous()):
        raise ValueError("y2 must be contiguous [T, d] (or [T * top, d]) in the dtype of y1, with its gate")
    if top and (row_weight is None or row_weight.dtype != torch.float32 or row_weight.shape != (T, top)
                or slot_to_row.dtype != torch.int32 or not row_weight.is_contiguous() or not slot_to_row.is_contiguous()):
        raise ValueError("row_weight must be fp32 and slot_to_row int32, both contiguous [T, top]")
    h = torch.empty(T, d, dtype=y1.dtype, device=x.device)
    check(lib.b200_gated_residual(x.data_ptr(), y1.data_ptr(), gate1.data_ptr(), _ptr(y2), _ptr(gate2), gate1.stride(0),
                                  _ptr(row_weight), _ptr(slot_to_row), top, h.data_ptr(), T, d, _dt(h),
                                  status_word(dev).data_ptr(), _stream()), "gated_residual")
    return h


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 per row of z [T, W] (row stride free), N a division by the root mean square."""
    _cuda(z, coef)
    _f32vec("coef", coef, 4)
    if z.stride(1) != 1:
        raise ValueError("rows must be contiguous")
    out = torch.empty(z.shape, dtype=z.dtype, device=z.device)
    check(lib.b200_poly_norm(z.data_ptr(), z.stride(0), coef.data_ptr(), float(eps), out.data_ptr(), z.shape[0], z.shape[1],
                             _dt(z), _stream()), "poly_norm")
    return out


def gelu_table(u: torch.Tensor, table: torch.Tensor, first: int, tokens: torch.Tensor) -> torch.Tensor:
    """gelu_tanh(u[t]) * table[tokens[t], first : first + W] for u [T, W], table [vocab, >= first + W]."""
    dev = _cuda(u, table, tokens)
    T, W = u.shape
    if not u.is_contiguous() or not table.is_contiguous() or table.dtype != u.dtype or first + W > table.shape[1]:
        raise ValueError("u and table must be contiguous, of one dtype, the table wide enough")
    _tokens("tokens", tokens, T)
    out = torch.empty_like(u)
    check(lib.b200_gelu_table(u.data_ptr(), table.data_ptr(), table.shape[1], table.shape[0], int(first), tokens.data_ptr(),
                              out.data_ptr(), T, W, _dt(u), status_word(dev).data_ptr(), _stream()), "gelu_table")
    return out


class Rotation:
    """Interleaved rotation of the first 2 * freq.numel() channels of a rotary part; cos and sin times ``magnitude``."""

    def __init__(self, base: float, dims: int, device, scaling: YarnScaling | None = None):
        self.dims = dims
        self.freq = rotary_frequencies(base, dims, device, scaling)
        self.magnitude = scaling.magnitude if scaling is not None else 1.0


def latent_prologue(q_in: torch.Tensor | None, q_norm_w: torch.Tensor | None, kv_in: torch.Tensor, kv_norm_w: torch.Tensor,
                    eps: float, rotation: Rotation, positions: torch.Tensor, cache: torch.Tensor, slot_mapping: torch.Tensor):
    """Norm of query latents [T, rq] and of latent rows [T, r | dr], whose last dr channels are rotated instead; the rows are
    also written to cache[slot_mapping] (``b200_latent_prologue``).  Inputs with free row strides.  Returns both."""
    dev = _cuda(q_in, q_norm_w, kv_in, kv_norm_w, rotation.freq, positions, cache, slot_mapping)
    T, W = kv_in.shape
    r = kv_norm_w.numel()
    _f32vec("kv_norm_w", kv_norm_w, r)
    if r > W or rotation.dims > W - r or kv_in.stride(1) != 1 or cache.shape[-1] != W or cache.dtype != kv_in.dtype \
            or not cache.is_contiguous():
        raise ValueError("latent rows / cache shape, dtype or layout mismatch")
    for name, t in (("positions", positions), ("slot_mapping", slot_mapping)):
        _tokens(name, t, T)
    q_out, rq = None, 0
    if q_in is not None:
        rq = q_in.shape[1]
        if q_in.shape[0] != T or q_in.stride(1) != 1 or q_in.dtype != kv_in.dtype:
            raise ValueError("query latents must be [T, rq] in the dtype of the latent rows")
        _f32vec("q_norm_w", q_norm_w, rq)
        q_out = torch.empty(T, rq, dtype=kv_in.dtype, device=kv_in.device)
    kv_out = torch.empty(T, W, dtype=kv_in.dtype, device=kv_in.device)
    check(lib.b200_latent_prologue(
        _ptr(q_in), q_in.stride(0) if q_in is not None else 0, _ptr(q_norm_w), rq, _ptr(q_out), kv_in.data_ptr(),
        kv_in.stride(0), kv_norm_w.data_ptr(), r, W - r, float(eps), rotation.freq.data_ptr(), rotation.dims,
        rotation.magnitude, positions.data_ptr(), kv_out.data_ptr(), cache.data_ptr(), slot_mapping.data_ptr(),
        cache.numel() // W, T, _dt(kv_in), status_word(dev).data_ptr(), _stream()), "latent_prologue")
    return q_out, kv_out


def rotate_heads(q: torch.Tensor, rope_dim: int, rotation: Rotation, positions: torch.Tensor, tail_rows: int = 0):
    """Rotates the last ``rope_dim`` channels of every head of q [T, H, D] in place; returns a contiguous copy of the rotated
    parts of the first ``tail_rows`` tokens [tail_rows, H, rope_dim] (None for none)."""
    _cuda(q, rotation.freq, positions)
    T, H, D = q.shape
    if not q.is_contiguous() or rope_dim > D or rotation.dims > rope_dim or tail_rows > T:
        raise ValueError("q must be contiguous [T, H, D] with the rotary part inside the head")
    _tokens("positions", positions, T)
    tail = torch.empty(tail_rows, H, rope_dim, dtype=q.dtype, device=q.device) if tail_rows else None
    check(lib.b200_rotate_heads(q.data_ptr(), T, H, D, rope_dim, rotation.freq.data_ptr(), rotation.dims, rotation.magnitude,
                                positions.data_ptr(), _ptr(tail), tail_rows, _dt(q), _stream()), "rotate_heads")
    return tail


def prefill_window_tile_rows(Hq: int, Hkv: int, Dqk: int, tail: int, Dv: int, dtype: torch.dtype) -> int:
    """Query rows per tile of the kernel behind ``prefill_varlen_window``; 0 = no tiled kernel."""
    return int(lib.b200_prefill_window_tile_rows(Hq, Hkv, Dqk, tail, Dv, _DTYPES[dtype])) if dtype in _DTYPES else 0


def prefill_varlen_window(q: torch.Tensor, k_head: torch.Tensor, k_tail: torch.Tensor | None, v: torch.Tensor,
                          cu_seqlens_q: torch.Tensor, cu_seqlens_k: torch.Tensor, max_seqlen_q: int, scale: float,
                          window: int = 0, sink: torch.Tensor | None = None, out: torch.Tensor | None = None,
                          plan: "PrefillPlan | None" = None) -> torch.Tensor:
    """Causal attention over packed keys [Tk, Hkv, Dqk - tail] with a part [Tk, tail] shared by the heads behind them (or
    None), a sliding window (0: none) and a sink (``b200_prefill_varlen_window``).  q [Tq, Hq, Dqk], v [Tk, Hkv, Dv]; token
    strides free, heads contiguous.  Contexts may start in the middle: only their ends count.  Returns [Tq, Hq, Dv]."""
    dev = _cuda(q, k_head, k_tail, v, cu_seqlens_q, cu_seqlens_k, sink, out)
    Tq, Hq, Dqk = q.shape
    Tk, Hkv, Dv = v.shape
    tail = k_tail.shape[1] if k_tail is not None else 0
    if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k.dtype != torch.int32 or cu_seqlens_q.numel() != cu_seqlens_k.numel():
        raise ValueError("cu_seqlens must be int32 tensors of the same length")
    if k_head.shape != (Tk, Hkv, Dqk - tail) or (tail and k_tail.shape[0] != Tk) \
            or any(t is not None and t.dtype != q.dtype for t in (k_head, k_tail, v)):
        raise ValueError("k_head must be [Tk, Hkv, Dqk - tail], k_tail [Tk, tail], v [Tk, Hkv, Dv] in the dtype of q")
    for t, D in ((q, Dqk), (k_head, Dqk - tail), (v, Dv)):
        if t.stride(2) != 1 or (t.shape[1] > 1 and t.stride(1) != D):
            raise ValueError("heads must be contiguous")
    if tail and k_tail.stride(1) != 1:
        raise ValueError("k_tail rows must be contiguous")
    _f32vec("sink", sink, Hq)
    if out is None:
        out = torch.empty((Tq, Hq, Dv), dtype=q.dtype, device=q.device)
    elif out.shape != (Tq, Hq, Dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [Tq, Hq, Dv] tensor")
    check(lib.b200_prefill_varlen_window(
        q.data_ptr(), k_head.data_ptr(), _ptr(k_tail), v.data_ptr(), out.data_ptr(), q.stride(0), k_head.stride(0),
        k_tail.stride(0) if tail else 0, v.stride(0), Tq, Tk, cu_seqlens_q.data_ptr(), cu_seqlens_k.data_ptr(),
        cu_seqlens_q.numel() - 1, int(max_seqlen_q), Hq, Hkv, Dqk, tail, Dv, float(scale), int(window), _ptr(sink),
        plan.buffer.data_ptr() if plan is not None else None, plan.tile_rows if plan is not None else 0,
        plan.capacity if plan is not None else 0, _dt(q), status_word(dev).data_ptr(), _stream()), "prefill_varlen_window")
    return out


def moe_group_route(logits: torch.Tensor, correction: torch.Tensor, top: int, groups: int = 1, keep: int = 1):
    """Grouped choice of ``top`` experts per token from fp32 logits [T, E] (``b200_moe_group_route``).  Returns (sorted_token
    [T * top], weight fp32 [T, top], expert_offsets [E], slot_to_row [T, top])."""
    dev = _cuda(logits, correction)
    T, E = logits.shape
    if logits.dtype != torch.float32 or not logits.is_contiguous():
        raise ValueError("logits must be contiguous fp32 [T, E]")
    _f32vec("correction", correction, E)
    tok = torch.empty(T * top, dtype=torch.int32, device=dev)
    w = torch.empty(T, top, dtype=torch.float32, device=dev)
    offs = torch.empty(E, dtype=torch.int32, device=dev)
    slot = torch.empty(T, top, dtype=torch.int32, device=dev)
    ws = workspace(dev, int(lib.b200_moe_group_route_workspace_bytes(T, E, top)), "moe_group_route")
    check(lib.b200_moe_group_route(logits.data_ptr(), correction.data_ptr(), T, E, int(top), int(groups), int(keep),
                                   tok.data_ptr(), w.data_ptr(), offs.data_ptr(), slot.data_ptr(), ws.data_ptr(), ws.numel(),
                                   _stream()), "moe_group_route")
    return tok, w, offs, slot


def moe_grouped_linear(x: torch.Tensor, w: torch.Tensor, expert_offsets: torch.Tensor,
                       glu: tuple[float, float] | None = None, early_launch: bool = False,
                       squared_relu: bool = False) -> torch.Tensor:
    """Rows of x [R, k] grouped by expert times the expert's weight w [E, n, k] -> [R, n], any size, bf16 or fp32.  ``glu``
    (limit, slope): w is [E, 2 n, k] = [gate | up] and the clamped gated unit of the two comes back [R, n]; ``squared_relu``:
    max(., 0)^2 of the result."""
    dev = _cuda(x, w, expert_offsets)
    (R, k), (E, n, k2) = x.shape, w.shape
    if x.dtype != w.dtype or k != k2 or not x.is_contiguous() or not w.is_contiguous() or expert_offsets.dtype != torch.int32 \
            or expert_offsets.numel() != E or (glu is not None and (n % 2 or squared_relu)):
        raise ValueError("x [R, k] and w [E, n, k] must be contiguous, of one dtype; expert_offsets int32 [E]")
    n_out = n // 2 if glu is not None else n
    limit, slope = glu if glu is not None else (0.0, 0.0)
    out = torch.empty(R, n_out, dtype=x.dtype, device=dev)
    check(lib.b200_moe_grouped_linear(x.data_ptr(), w.data_ptr(), out.data_ptr(), expert_offsets.data_ptr(), R, E, n_out, k,
                                      1 if glu is not None else 2 if squared_relu else 0, float(limit), float(slope),
                                      MOE_GEMM_EARLY_LAUNCH if early_launch else 0, _dt(x), status_word(dev).data_ptr(),
                                      _stream()), "moe_grouped_linear")
    return out


# ------------------------------------------------------------------------------------------------
# token shift, convolved queries and keys, sigmoid attention in chunks, softmax over the chosen experts
# ------------------------------------------------------------------------------------------------
@dataclass
class StepRows:
    """Which sequence the rows of a step belong to, for kernels that carry state from token to token: ragged portions
    (``cu_seqlens_q`` / ``cu_seqlens_k``), or row i = sequence i with ``context_lens`` tokens."""
    state_slots: torch.Tensor                     # int64 [n], -1 = no state
    cu_seqlens_q: torch.Tensor | None = None      # int32 [n + 1]
    cu_seqlens_k: torch.Tensor | None = None
    context_lens: torch.Tensor | None = None      # int64 [n]

    @classmethod
    def of(cls, ctx) -> "StepRows":
        if ctx.is_prefill:
            return cls(ctx.state_slots, ctx.cu_seqlens_q, ctx.cu_seqlens_k)
        return cls(ctx.state_slots, context_lens=ctx.context_lens)

    def check(self, T: int) -> int:
        """Number of sequences."""
        ragged = self.cu_seqlens_q is not None
        n = self.cu_seqlens_q.numel() - 1 if ragged else T
        if self.state_slots.dtype != torch.int64 or self.state_slots.numel() < n or not self.state_slots.is_contiguous():
            raise ValueError("state_slots must be contiguous int64 with one entry per sequence")
        if ragged:
            if self.cu_seqlens_q.dtype != torch.int32 or self.cu_seqlens_k is None or self.cu_seqlens_k.dtype != torch.int32 \
                    or self.cu_seqlens_k.numel() != n + 1:
                raise ValueError("cu_seqlens must be int32 tensors of the same length")
        elif self.context_lens is None or self.context_lens.dtype != torch.int64 or self.context_lens.numel() != T \
                or not self.context_lens.is_contiguous():
            raise ValueError("context_lens must be contiguous int64 with one entry per row")
        return n


def shift_residual(x: torch.Tensor | None, eps: float, dtype: torch.dtype, *, x_out: torch.Tensor | None = None,
                   tokens: torch.Tensor | None = None, embed: torch.Tensor | None = None, embed_scale: float = 1.0,
                   y: torch.Tensor | None = None, gain: float = 1.0, row_weight: torch.Tensor | None = None,
                   slot_to_row: torch.Tensor | None = None, shift: torch.Tensor | None = None,
                   state: torch.Tensor | None = None, rows: StepRows | None = None,
                   final_gain: float | None = None) -> torch.Tensor:
    """One boundary of a residual x [T, d] fp32 (``b200_shift_residual``): x' = x + gain y / rms(y), with y dense [T, d] or
    the expert rows [T * top, d] behind ``slot_to_row`` / ``row_weight`` [T, top], or x' = the scaled embedding rows.  x' goes to
    ``x_out``.  Returns x' in ``dtype``, mixed with the previous token's (``shift`` [d], ``state`` [slots, d], ``rows``), or
    normed with one number (``final_gain``)."""
    dev = _cuda(x, x_out, tokens, embed, y, row_weight, slot_to_row, shift, state)
    T, d = (tokens.numel(), embed.shape[1]) if embed is not None else x.shape
    for name, t in (("x", x if embed is None else None), ("x_out", x_out)):
        if t is not None and (t.dtype != torch.float32 or t.shape != (T, d) or not t.is_contiguous()):
            raise ValueError(f"{name} must be a contiguous fp32 [T, d] tensor")
    if embed is not None:
        if embed.dtype != dtype or not embed.is_contiguous():
            raise ValueError("embed must be contiguous [vocab, d] in the activation dtype")
        _tokens("tokens", tokens, T)
    top = slot_to_row.shape[1] if slot_to_row is not None else 0
    if y is not None and (y.shape != ((T * top) if top else T, d) or y.dtype != dtype or not y.is_contiguous()):
        raise ValueError("y must be contiguous [T, d] (or [T * top, d]) in the activation dtype")
    if top and (y is None or row_weight is None or row_weight.dtype != torch.float32 or row_weight.shape != (T, top)
                or slot_to_row.dtype != torch.int32 or not row_weight.is_contiguous() or not slot_to_row.is_contiguous()):
        raise ValueError("row_weight must be fp32 and slot_to_row int32, both contiguous [T, top]")
    n = 0
    if shift is not None:
        _f32vec("shift", shift, d)
        if state is None or state.dtype != torch.float32 or state.dim() != 2 or state.shape[1] != d or not state.is_contiguous():
            raise ValueError("state must be contiguous fp32 [slots, d]")
        if x is not None and x_out is not None and x.data_ptr() == x_out.data_ptr() and embed is None:
            raise ValueError("with a shift the residual cannot be updated in place")
        n = rows.check(T)
    h = torch.empty(T, d, dtype=dtype, device=dev)
    check(lib.b200_shift_residual(
        _ptr(x), _ptr(x_out), _ptr(tokens) if embed is not None else None, _ptr(embed), embed.shape[0] if embed is not None else 0,
        float(embed_scale), _ptr(y), _ptr(row_weight), _ptr(slot_to_row), top, float(gain), _ptr(shift), _ptr(state),
        state.shape[0] if state is not None else 0, rows.state_slots.data_ptr() if shift is not None else None,
        _ptr(rows.cu_seqlens_q) if shift is not None else None, _ptr(rows.cu_seqlens_k) if shift is not None else None,
        _ptr(rows.context_lens) if shift is not None else None, n, 1 if final_gain is not None else 0, float(final_gain or 0.0),
        float(eps), h.data_ptr(), T, d, _dt(h), status_word(dev).data_ptr(), _stream()), "shift_residual")
    return h


def conv_norm_rope_store(q: torch.Tensor, k: torch.Tensor, conv_q: torch.Tensor, conv_k: torch.Tensor,
                         ring: torch.Tensor | None, rows: StepRows, q_norm_w: torch.Tensor, k_norm_w: torch.Tensor, eps: float,
                         freq: torch.Tensor, positions: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor,
                         slot_mapping: torch.Tensor, packed: bool = True):
    """Short convolution of q [T, Hq * D] and k [T, Hkv * D] (views of one projection; weights [taps, channels]), values = the
    convolved keys, norms over the whole projections, rotation of channel halves, scatter into the pools [num_blocks,
    block_size, Hkv, D] (``b200_conv_norm_rope_store``).  ``ring`` [slots, taps - 1, channels of q and k] carries the last inputs.
    Returns q [T, Hq, D] and, with ``packed``, k and v [T, Hkv, D] (else None)."""
    dev = _cuda(q, k, conv_q, conv_k, ring, q_norm_w, k_norm_w, freq, positions, k_cache, v_cache, slot_mapping)
    nb, bs, Hkv, D = k_cache.shape
    T, taps = q.shape[0], conv_q.shape[0]
    Cq, Ck = q.shape[1], Hkv * D
    if Cq % D or k.shape != (T, Ck) or any(t.stride(1) != 1 or t.stride(0) != q.stride(0) or t.dtype != q.dtype for t in (q, k)):
        raise ValueError("q [T, Hq * D] and k [T, Hkv * D] must share dtype and row stride")
    if v_cache.shape != k_cache.shape or any(not c.is_contiguous() or c.dtype != q.dtype for c in (k_cache, v_cache)):
        raise ValueError("caches must be contiguous [num_blocks, block_size, Hkv, D] of q's dtype")
    _f32vec("conv_q", conv_q, taps * Cq)
    _f32vec("conv_k", conv_k, taps * Ck)
    _f32vec("q_norm_w", q_norm_w, Cq)
    _f32vec("k_norm_w", k_norm_w, Ck)
    if taps > 1 and (ring is None or ring.dtype != torch.float32 or ring.shape[1:] != (taps - 1, Cq + Ck) or not ring.is_contiguous()):
        raise ValueError("ring must be contiguous fp32 [slots, taps - 1, channels]")
    if freq.dtype != torch.float64 or not freq.is_contiguous():
        raise ValueError("freq must be contiguous fp64")
    for name, t in (("positions", positions), ("slot_mapping", slot_mapping)):
        _tokens(name, t, T)
    n = rows.check(T)
    qo = torch.empty(T, Cq // D, D, dtype=q.dtype, device=dev)
    ko, vo = (torch.empty(T, Hkv, D, dtype=q.dtype, device=dev) for _ in range(2)) if packed else (None, None)
    check(lib.b200_conv_norm_rope_store(
        q.data_ptr(), k.data_ptr(), q.stride(0), conv_q.data_ptr(), conv_k.data_ptr(), taps, _ptr(ring) if taps > 1 else None,
        ring.shape[0] if taps > 1 else 0, rows.state_slots.data_ptr(), _ptr(rows.cu_seqlens_q), _ptr(rows.cu_seqlens_k),
        _ptr(rows.context_lens), n, q_norm_w.data_ptr(), k_norm_w.data_ptr(), float(eps), freq.data_ptr(), 2 * freq.numel(),
        positions.data_ptr(), qo.data_ptr(), _ptr(ko), _ptr(vo), k_cache.data_ptr(), v_cache.data_ptr(), slot_mapping.data_ptr(),
        nb * bs, T, Cq // D, Hkv, D, _dt(q), status_word(dev).data_ptr(), _stream()), "conv_norm_rope_store")
    return qo, ko, vo


def sigmoid_attention_tile_rows(Hq: int, Hkv: int, Dqk: int, Dv: int, dtype: torch.dtype) -> int:
    """Query rows per tile of the kernel behind ``sigmoid_attention``; 0 = no tiled kernel."""
    return int(lib.b200_sigmoid_attention_tile_rows(Hq, Hkv, Dqk, Dv, _DTYPES[dtype])) if dtype in _DTYPES else 0


def _gate_rows(gate: torch.Tensor | None, rows: int, heads: int, dtype: torch.dtype) -> None:
    if gate is not None and (gate.shape != (rows, heads) or gate.dtype != dtype or (heads > 1 and gate.stride(1) != 1)):
        raise ValueError("gate must be [tokens, heads] in the dtype of q with contiguous rows")


def sigmoid_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, cu_seqlens_q: torch.Tensor, cu_seqlens_k: torch.Tensor,
                      max_seqlen_q: int, scale: float, bias: torch.Tensor, chunk: int = 0, gate: torch.Tensor | None = None,
                      out: torch.Tensor | None = None, plan: "PrefillPlan | None" = None) -> torch.Tensor:
    """Causal attention over packed keys with weights sigmoid(scale q.k + bias[head]), not normalised, inside chunks of
    positions (0: none), every head's row times sigmoid(gate) (``b200_sigmoid_attention``).  q [Tq, Hq, Dqk], k [Tk, Hkv, Dqk],
    v [Tk, Hkv, Dv]; packed contexts start where a chunk starts.  Returns [Tq, Hq, Dv]."""
    dev = _cuda(q, k, v, cu_seqlens_q, cu_seqlens_k, bias, gate, out)
    Tq, Hq, Dqk = q.shape
    Tk, Hkv, Dv = v.shape
    if cu_seqlens_q.dtype != torch.int32 or cu_seqlens_k.dtype != torch.int32 or cu_seqlens_q.numel() != cu_seqlens_k.numel():
        raise ValueError("cu_seqlens must be int32 tensors of the same length")
    if k.shape != (Tk, Hkv, Dqk) or k.dtype != q.dtype or v.dtype != q.dtype:
        raise ValueError("k must be [Tk, Hkv, Dqk] and v [Tk, Hkv, Dv] in the dtype of q")
    for t, D in ((q, Dqk), (k, Dqk), (v, Dv)):
        if t.stride(2) != 1 or (t.shape[1] > 1 and t.stride(1) != D):
            raise ValueError("heads must be contiguous")
    _f32vec("bias", bias, Hq)
    _gate_rows(gate, Tq, Hq, q.dtype)
    if out is None:
        out = torch.empty((Tq, Hq, Dv), dtype=q.dtype, device=q.device)
    elif out.shape != (Tq, Hq, Dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [Tq, Hq, Dv] tensor")
    check(lib.b200_sigmoid_attention(
        q.data_ptr(), k.data_ptr(), v.data_ptr(), out.data_ptr(), q.stride(0), k.stride(0), v.stride(0), Tq, Tk,
        cu_seqlens_q.data_ptr(), cu_seqlens_k.data_ptr(), cu_seqlens_q.numel() - 1, int(max_seqlen_q), Hq, Hkv, Dqk, Dv,
        float(scale), bias.data_ptr(), int(chunk), _ptr(gate), gate.stride(0) if gate is not None else 0,
        plan.buffer.data_ptr() if plan is not None else None, plan.tile_rows if plan is not None else 0,
        plan.capacity if plan is not None else 0, _dt(q), status_word(dev).data_ptr(), _stream()), "sigmoid_attention")
    return out


def sigmoid_decode(q: torch.Tensor, k_cache: torch.Tensor, v_cache: torch.Tensor, block_tables: torch.Tensor,
                   context_lens: torch.Tensor, scale: float, bias: torch.Tensor, chunk: int = 0, gate: torch.Tensor | None = None,
                   out: torch.Tensor | None = None) -> torch.Tensor:
    """``sigmoid_attention`` of one token per sequence over the paged pools (``b200_sigmoid_decode``): q [B, Hq, D], caches
    [num_blocks, block_size, Hkv, D*].  Returns [B, Hq, Dv]."""
    dev = _cuda(q, k_cache, v_cache, block_tables, context_lens, bias, gate, out)
    B, Hq, D = q.shape
    nb, bs, Hkv, Dc = k_cache.shape
    Dv = v_cache.shape[3]
    if Dc != D or v_cache.shape[:3] != k_cache.shape[:3] or k_cache.dtype != q.dtype or v_cache.dtype != q.dtype \
            or not (q.is_contiguous() and k_cache.is_contiguous() and v_cache.is_contiguous()):
        raise ValueError("q and caches must be contiguous, of one dtype and head size")
    if block_tables.dtype != torch.int32 or block_tables.dim() != 2 or block_tables.shape[0] != B or block_tables.stride(1) != 1 \
            or context_lens.dtype != torch.int64 or context_lens.numel() != B or not context_lens.is_contiguous():
        raise ValueError("block_tables must be int32 [B, maxb] and context_lens int64 [B]")
    _f32vec("bias", bias, Hq)
    _gate_rows(gate, B, Hq, q.dtype)
    if out is None:
        out = torch.empty((B, Hq, Dv), dtype=q.dtype, device=q.device)
    elif out.shape != (B, Hq, Dv) or out.dtype != q.dtype or not out.is_contiguous():
        raise ValueError("out must be a contiguous [B, Hq, Dv] tensor of q's dtype")
    ws = workspace(dev, lib.b200_paged_decode_gqa_workspace_bytes(B, Hq, Hkv, D, _dt(q)), "decode")
    check(lib.b200_sigmoid_decode(
        q.data_ptr(), k_cache.data_ptr(), v_cache.data_ptr(), out.data_ptr(), block_tables.data_ptr(), block_tables.stride(0),
        context_lens.data_ptr(), B, Hq, Hkv, D, Dv, bs, nb, float(scale), bias.data_ptr(), int(chunk), _ptr(gate),
        gate.stride(0) if gate is not None else 0, ws.data_ptr(), ws.numel(), _dt(q), status_word(dev).data_ptr(), _stream()),
        "sigmoid_decode")
    return out


def moe_softmax_route(logits: torch.Tensor, bias: torch.Tensor, top: int):
    """The ``top`` experts with the largest logits + bias per token, weights = softmax over those alone; fp32 logits [T, E]
    (``b200_moe_softmax_route``).  Returns what ``moe_group_route`` returns."""
    dev = _cuda(logits, bias)
    T, E = logits.shape
    if logits.dtype != torch.float32 or not logits.is_contiguous():
        raise ValueError("logits must be contiguous fp32 [T, E]")
    _f32vec("bias", bias, E)
    tok = torch.empty(T * top, dtype=torch.int32, device=dev)
    w = torch.empty(T, top, dtype=torch.float32, device=dev)
    offs = torch.empty(E, dtype=torch.int32, device=dev)
    slot = torch.empty(T, top, dtype=torch.int32, device=dev)
    ws = workspace(dev, int(lib.b200_moe_group_route_workspace_bytes(T, E, top)), "moe_group_route")
    check(lib.b200_moe_softmax_route(logits.data_ptr(), bias.data_ptr(), T, E, int(top), tok.data_ptr(), w.data_ptr(),
                                     offs.data_ptr(), slot.data_ptr(), ws.data_ptr(), ws.numel(), _stream()), "moe_softmax_route")
    return tok, w, offs, slot
