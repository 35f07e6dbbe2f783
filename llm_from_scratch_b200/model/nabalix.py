"""The Nabalix decoder family: hyper-connected residual streams around a parallel mixer (gated talking-heads
window attention beside an HGRN2 recurrence) and an optional clamped GLU, every layer with its own sizes.

The module only composes mechanisms of ``mixers`` and the shared head; caches, batching and sampling are the
engine's.  Parameter names are those of the family's checkpoints (``l<i>.mix.left.q`` and so on).  The residual
streams, norms, scores, gates and states are fp32 in either compute dtype; matrix products and activations
between them are in the compute dtype.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .mixers import ClampedGLU, GatedRecurrence, HyperConnection, Params, ParallelMixer, TalkingHeadsAttention
from .registry import ModelFamily, register
from .transformer import TokenHead


@dataclass
class NabalixLayer:
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    softcap: float
    window: int                       # 0: no window
    rec_heads: int
    rec_dim: int
    rec_vdim: int
    d_ff: int = 0                     # 0: no feed-forward
    limit: float = 0.0

    @classmethod
    def from_dict(cls, d: dict) -> "NabalixLayer":
        if d["type"] != "parallel":
            raise ValueError(f"unsupported mixer type {d['type']!r}")
        left, right, mlp = d["mixer"]["left"], d["mixer"]["right"], d.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
        layer = cls(heads=left["heads"], kv_heads=left["kv_heads"], dim=left["dim"], vdim=left["vdim"],
                    scale=float(left["scale"]), softcap=float(left.get("softcap") or 0.0),
                    window=int((left.get("mask") or {}).get("size") or 0), rec_heads=right["heads"],
                    rec_dim=right["dim"], rec_vdim=right["vdim"], d_ff=mlp["ff"] if mlp else 0,
                    limit=float(mlp["limit"]) if mlp else 0.0)
        if layer.heads % layer.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        return layer

    def to_dict(self) -> dict:
        return {"type": "parallel",
                "mixer": {"left": {"heads": self.heads, "kv_heads": self.kv_heads, "dim": self.dim, "vdim": self.vdim,
                                   "scale": self.scale, "softcap": self.softcap, "mask": {"size": self.window}},
                          "right": {"heads": self.rec_heads, "dim": self.rec_dim, "vdim": self.rec_vdim}},
                "mlp": {"kind": "dense", "ff": self.d_ff, "limit": self.limit} if self.d_ff else None}


@dataclass
class NabalixConfig:
    vocab_size: int
    d_model: int
    streams: int
    eps: float
    layers: list = field(default_factory=list)
    context_length: Optional[int] = None      # positions are unbounded; None = as long as the cache pool holds

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict) -> "NabalixConfig":
        return cls(vocab_size=d["vocab"], d_model=d["width"], streams=d.get("streams", 1), eps=float(d["norm"]["eps"]),
                   layers=[NabalixLayer.from_dict(x) for x in d["layers"]], context_length=d.get("context_length"))

    def to_dict(self) -> dict:
        out = {"architecture": "Nabalix", "vocab": self.vocab_size, "width": self.d_model, "streams": self.streams,
               "norm": {"eps": self.eps}, "layers": [x.to_dict() for x in self.layers]}
        if self.context_length is not None:
            out["context_length"] = self.context_length
        return out


class NabalixBlock(nn.Module):
    def __init__(self, p: Params, cfg: NabalixConfig, c: NabalixLayer):
        super().__init__()
        d, eps = cfg.d_model, cfg.eps
        m = p.at("mix.")
        self.mixer = ParallelMixer(
            m, d, TalkingHeadsAttention(m.at("left."), d, c.heads, c.kv_heads, c.dim, c.vdim, c.scale, c.softcap, c.window),
            GatedRecurrence(m.at("right."), d, c.rec_heads, c.rec_dim, c.rec_vdim, eps))
        # (sublayer, its connection to the streams, norm weights of the join of its two results)
        self.sublayers = [(self.mixer, HyperConnection(p, 1, d, cfg.streams), self.mixer.join)]
        if c.d_ff:
            self.mlp = ClampedGLU(p.at("mlp."), d, c.d_ff, c.limit)
            self.sublayers.append((self.mlp, HyperConnection(p, 2, d, cfg.streams), None))


class NabalixLM(TokenHead, nn.Module):
    """``model(input_ids)`` -> final-norm hidden states [T, d]; the head is the one all models of the engine share."""

    # what the engine needs to know (engine/model_runner.py, engine/llm_engine.py)
    recurrent_state = True      # per-sequence state slots; no prefix reuse
    mixed_batches = True        # portions of prompts and decoded tokens share a step; keys always come from the pool

    def __init__(self, cfg: NabalixConfig, weights: dict, device, dtype=torch.float32):
        super().__init__()
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        p = Params(weights, self.device, dtype)
        self.embed = p.lin("embed", (cfg.vocab_size, cfg.d_model))
        self.layers = nn.ModuleList([NabalixBlock(p.at(f"l{i}."), cfg, c) for i, c in enumerate(cfg.layers)])
        self.final_norm = p.f32("final.norm", (cfg.d_model,))
        self.w_head, self.b_head = p.lin("head", (cfg.vocab_size, cfg.d_model)), None
        self.sublayers = [s for layer in self.layers for s in layer.sublayers]

    def cache_owners(self):
        """Modules with pools to allocate, layer by layer."""
        return [m for layer in self.layers for m in (layer.mixer.left, layer.mixer.right)]

    def prefill_tile_rows(self) -> int:
        return ops.TALKING_TILE_ROWS if self.dtype == torch.bfloat16 else 0

    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor | None = None) -> torch.Tensor:
        ctx, cfg = get_context(), self.cfg
        x = torch.empty(input_ids.shape[0], cfg.streams, cfg.d_model, dtype=torch.float32, device=input_ids.device)
        args = dict(tokens=input_ids, embed=self.embed)      # the first boundary starts the streams
        for sub, hc, join in self.sublayers:
            h = ops.stream_update(x, hc.norm, cfg.eps, self.dtype, in_w=hc.read, **args)
            y, y1 = sub(h, ctx)
            args = dict(y=y, y1=y1, join_w=join, join_eps=cfg.eps, layer_scale=hc.scale, mix=hc.mix, out_w=hc.write)
        return ops.stream_update(x, self.final_norm, cfg.eps, self.dtype, **args)


@torch.no_grad()
def init_weights(cfg: NabalixConfig, seed: int = 0, dtype=torch.float32) -> dict[str, torch.Tensor]:
    """Random parameters of the family's shapes under its checkpoint names (weights to run or test with, not a
    published initialisation): matrices N(0, 1/fan_in), gates that mostly keep, a head mix near the identity."""
    g = torch.Generator().manual_seed(seed)
    d, S = cfg.d_model, cfg.streams
    w: dict[str, torch.Tensor] = {}

    def lin(name, n, k):
        w[name] = (torch.randn(n, k, generator=g) * k ** -0.5).to(dtype)

    def vec(name, n, mean, std):
        w[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    w["embed"] = torch.randn(cfg.vocab_size, d, generator=g).to(dtype)
    for i, c in enumerate(cfg.layers):
        p = f"l{i}."
        left, right = p + "mix.left.", p + "mix.right."
        lin(left + "q", c.heads * c.dim, d)
        lin(left + "k", c.kv_heads * c.dim, d)
        lin(left + "v", c.kv_heads * c.vdim, d)
        lin(left + "g", c.heads * c.vdim, d)
        lin(left + "o", d, c.heads * c.vdim)
        w[left + "r1"] = torch.rand(c.heads, generator=g).to(dtype)
        w[left + "r2"] = torch.rand(c.heads, generator=g).to(dtype)
        w[left + "talk"] = (torch.eye(c.heads) + 0.2 * torch.randn(c.heads, c.heads, generator=g)).to(dtype)
        lin(right + "q", c.rec_heads * c.rec_dim, d)
        lin(right + "f", c.rec_heads * c.rec_dim, d)
        vec(right + "f.b", c.rec_heads * c.rec_dim, 3.0, 1.5)
        w[right + "lower"] = (0.9 * torch.rand(c.rec_heads * c.rec_dim, generator=g)).to(dtype)
        lin(right + "v", c.rec_heads * c.rec_vdim, d)
        vec(right + "norm", c.rec_vdim, 1.0, 0.1)
        lin(right + "o", d, c.rec_heads * c.rec_vdim)
        vec(left + "out", d, 1.0, 0.1)
        vec(right + "out", d, 1.0, 0.1)
        for q in (1, 2) if c.d_ff else (1,):
            vec(p + f"norm{q}", d, 0.0, 0.1)
            vec(p + f"ls{q}", d, 0.7, 0.1)
            vec(p + f"hc{q}.in", S, 1.0 / S, 0.1)
            vec(p + f"hc{q}.out", S, 1.0, 0.1)
            w[p + f"hc{q}.mix"] = (torch.eye(S) + 0.1 * torch.randn(S, S, generator=g)).to(dtype)
        if c.d_ff:
            lin(p + "mlp.gate", c.d_ff, d)
            lin(p + "mlp.up", c.d_ff, d)
            lin(p + "mlp.down", d, c.d_ff)
    vec("final.norm", d, 0.0, 0.1)
    lin("head", cfg.vocab_size, d)
    return w


register(ModelFamily("Nabalix", NabalixConfig, NabalixLM, init_weights))
