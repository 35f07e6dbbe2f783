"""The Sodonex decoder family: sigmoid attention inside chunks of positions over convolved queries and keys, inputs shifted by one
token, squared-ReLU experts behind a softmax over the chosen ones, and norms with one number on what the sublayers give.

The module only composes mechanisms of ``mixers`` and the shared head; caches, batching and sampling are the engine's.
Parameter names are those of the family's checkpoints (``l<i>.mix.q`` and so on).  The residual with its shift, norms, angles,
scores, attention weights and router are fp32 in either compute dtype; matrix products and activations between them are in the
compute dtype.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .mixers import Params, SigmoidAttention, SoftmaxMoE, TokenShift
from .registry import ModelFamily, register
from .transformer import TokenHead


@dataclass
class SodonexLayer:
    heads: int
    kv_heads: int
    dim: int                          # of queries, keys and values
    conv: int                         # taps
    scale: float
    rot_dims: int = 0
    rot_base: float = 10000.0
    chunk: int = 0                    # positions per chunk; 0: no chunks
    d_ff: int = 0                     # of every expert; 0: no feed-forward
    experts: int = 0
    top: int = 0

    @classmethod
    def from_dict(cls, d: dict) -> "SodonexLayer":
        if d["type"] != "attention":
            raise ValueError(f"unsupported mixer type {d['type']!r}")
        m, mlp = d["mixer"], d.get("mlp")
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        c = cls(heads=m["heads"], kv_heads=m["kv_heads"], dim=m["dim"], conv=m["conv"], scale=float(m["scale"]),
                rot_dims=int(rot.get("dims", 0)), rot_base=float(rot.get("base", 10000.0)), chunk=int(mask.get("size") or 0))
        if m.get("vdim", c.dim) != c.dim:
            raise ValueError("the values are the keys: dim and vdim must be equal")
        if c.heads % c.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        if c.rot_dims % 2 or c.rot_dims > c.dim:
            raise ValueError("rotated channels come in pairs inside the head")
        if c.conv < 1:
            raise ValueError("the convolution has at least one tap")
        if mlp is None:
            return c
        if mlp["kind"] != "moe":
            raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
        c.d_ff, c.experts, c.top = mlp["expert"]["ff"], mlp["router"]["experts"], mlp["router"]["top"]
        if not 0 < c.top <= c.experts:
            raise ValueError("a token uses at least one expert and at most all of them")
        return c

    def to_dict(self) -> dict:
        mixer = dict(heads=self.heads, kv_heads=self.kv_heads, dim=self.dim, vdim=self.dim, conv=self.conv, scale=self.scale,
                     rot={"dims": self.rot_dims, "base": self.rot_base}, mask={"size": self.chunk} if self.chunk else None)
        mlp = None
        if self.experts:
            mlp = {"kind": "moe", "expert": {"ff": self.d_ff}, "router": {"experts": self.experts, "top": self.top}}
        return {"type": "attention", "mixer": mixer, "mlp": mlp}


@dataclass
class SodonexConfig:
    vocab_size: int
    d_model: int
    eps: float
    embed_scale: float
    residual_mult: float                      # of what a sublayer adds to the residual
    layers: list = field(default_factory=list)
    context_length: Optional[int] = None      # positions are unbounded; None = as long as the cache pool holds

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict) -> "SodonexConfig":
        return cls(vocab_size=d["vocab"], d_model=d["width"], eps=float(d["norm"]["eps"]),
                   embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)), residual_mult=float(d.get("residual_mult", 1.0)),
                   layers=[SodonexLayer.from_dict(x) for x in d["layers"]], context_length=d.get("context_length"))

    def to_dict(self) -> dict:
        out = {"architecture": "Sodonex", "vocab": self.vocab_size, "width": self.d_model, "norm": {"eps": self.eps},
               "embedding": {"scale": self.embed_scale}, "residual_mult": self.residual_mult,
               "layers": [x.to_dict() for x in self.layers]}
        if self.context_length is not None:
            out["context_length"] = self.context_length
        return out


def _number(p: Params, name: str) -> float:
    t = p.raw(name)
    if t.numel() != 1:
        raise ValueError(f"{p.prefix + name} must be a single number, not {tuple(t.shape)}")
    return float(t)


class SodonexBlock(nn.Module):
    def __init__(self, p: Params, cfg: SodonexConfig, c: SodonexLayer):
        super().__init__()
        d = cfg.d_model
        self.shift = TokenShift(p, d)
        self.mixer = SigmoidAttention(p.at("mix."), d, c.heads, c.kv_heads, c.dim, c.conv, c.scale, c.rot_dims, c.rot_base, c.chunk,
                                      cfg.eps)
        # what the sublayers' normed results are multiplied by on their way into the residual
        self.gain1 = cfg.residual_mult * _number(p, "norm1")
        self.mlp, self.gain2 = None, 0.0
        if c.experts:
            self.mlp = SoftmaxMoE(p.at("mlp."), d, c.d_ff, c.experts, c.top)
            self.gain2 = cfg.residual_mult * _number(p, "norm2")


class SodonexLM(TokenHead, nn.Module):
    """``model(input_ids)`` -> final-norm hidden states [T, d]; the head is the one all models of the engine share."""

    # what the engine needs to know (engine/model_runner.py, engine/llm_engine.py)
    recurrent_state = True      # slots for the last token and the convolutions' last inputs of every sequence
    mixed_batches = True        # portions of prompts and decoded tokens share a step
    splits_steps = True         # ... and the single tokens of such a step run on the decode kernels

    def __init__(self, cfg: SodonexConfig, weights: dict, device, dtype=torch.float32):
        super().__init__()
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        p = Params(weights, self.device, dtype)
        self.embed = p.lin("embed", (cfg.vocab_size, cfg.d_model))
        self.layers = nn.ModuleList([SodonexBlock(p.at(f"l{i}."), cfg, c) for i, c in enumerate(cfg.layers)])
        self.final_gain = _number(p, "final.norm")
        self.w_head, self.b_head = p.lin("head", (cfg.vocab_size, cfg.d_model)), None
        # steps of whole prompts can be captured: every layer's attention then takes its grid from a tile list
        self.captures_prompts = all(layer.mixer.tile_rows(dtype) for layer in self.layers)
        self.attention_chunks = sorted({c.chunk for c in cfg.layers if c.chunk})

    def cache_owners(self):
        """Modules with pools to allocate, layer by layer."""
        return [m for layer in self.layers for m in (layer.shift, layer.mixer)]

    def prefill_tile_rows(self) -> int:
        return 0        # the layers ask for the tile lists they need (Portions.plan)

    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor | None = None) -> torch.Tensor:
        ctx, cfg = get_context(), self.cfg
        if positions is None:
            positions = ctx.positions if ctx.positions is not None else ctx.context_lens - 1
        rows = ops.StepRows.of(ctx)
        # the residual, and the buffer it moves to at every shift
        x, spare = (torch.empty(input_ids.shape[0], cfg.d_model, dtype=torch.float32, device=input_ids.device) for _ in range(2))
        step = dict(tokens=input_ids, embed=self.embed, embed_scale=cfg.embed_scale)
        for layer in self.layers:
            h = ops.shift_residual(x, cfg.eps, self.dtype, x_out=spare, shift=layer.shift.weight, state=layer.shift.state, rows=rows,
                                   **step)
            x, spare = spare, x
            step = dict(y=layer.mixer(h, ctx, positions, rows), gain=layer.gain1)
            if layer.mlp is not None:
                f, weight, slot = layer.mlp(ops.shift_residual(x, cfg.eps, self.dtype, x_out=x, **step))
                step = dict(y=f, row_weight=weight, slot_to_row=slot, gain=layer.gain2)
        return ops.shift_residual(x, cfg.eps, self.dtype, final_gain=self.final_gain, **step)

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.logits_f32(hidden)


@torch.no_grad()
def init_weights(cfg: SodonexConfig, seed: int = 0, dtype=torch.float32) -> dict[str, torch.Tensor]:
    """Random parameters of the family's shapes under its checkpoint names (weights to run or test with, not a published
    initialisation): matrices N(0, 1/fan_in), convolutions N(0, 1/taps), attention weights around one tenth, mild shifts."""
    g = torch.Generator().manual_seed(seed)
    d = cfg.d_model
    w: dict[str, torch.Tensor] = {}

    def lin(name, n, k):
        w[name] = (torch.randn(n, k, generator=g) * k ** -0.5).to(dtype)

    def vec(name, n, mean, std):
        w[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    def number(name, mean, std):
        w[name] = (mean + std * torch.randn((), generator=g)).to(dtype)

    w["embed"] = torch.randn(cfg.vocab_size, d, generator=g).to(dtype)
    for i, c in enumerate(cfg.layers):
        p, m = f"l{i}.", f"l{i}.mix."
        w[p + "shift"] = (0.6 * torch.rand(d, generator=g)).to(dtype)
        for name, n in (("q", c.heads * c.dim), ("k", c.kv_heads * c.dim)):
            lin(m + name, n, d)
            vec(m + name + ".b", n, 0.0, 0.3)
            w[m + name + ".conv"] = (torch.randn(n, c.conv, generator=g) * c.conv ** -0.5).to(dtype)
            vec(m + name + ".norm", n, 1.0, 0.2)
        vec(m + "pb", c.heads, -2.0, 0.7)
        lin(m + "g", c.heads, d)
        lin(m + "o", d, c.heads * c.dim)
        vec(m + "o.b", d, 0.0, 0.1)
        number(p + "norm1", 1.0, 0.1)
        if c.experts:
            lin(p + "mlp.router", c.experts, d)
            vec(p + "mlp.router.b", c.experts, 0.0, 0.5)
            for e in range(c.experts):
                lin(f"{p}mlp.e{e}.up", c.d_ff, d)
                lin(f"{p}mlp.e{e}.down", d, c.d_ff)
            number(p + "norm2", 1.0, 0.1)
    number("final.norm", 1.0, 0.1)
    lin("head", cfg.vocab_size, d)
    return w


register(ModelFamily("Sodonex", SodonexConfig, SodonexLM, init_weights))
