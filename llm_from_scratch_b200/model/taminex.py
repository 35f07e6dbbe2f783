"""The Taminex decoder family: an fp32 residual whose layers norm the sublayer's output, with three kinds of mixer in any
order — gated delta rule, latent attention without positions (layers may share latent rows), attention with sinks and
interleaved rotation — squared-ReLU feed-forwards and a tied, scaled, soft-capped head.

The module only composes mechanisms of ``mixers`` and the shared head; caches, batching and sampling are the engine's.
Parameter names are those of the family's checkpoints (``l<i>.mix.q`` and so on).  The residual, norms, angles, scores, gates
of the recurrence and states are fp32 in either compute dtype; matrix products and activations between them are in the
compute dtype.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .mixers import GatedDeltaRule, LatentAttention, Params, SinkAttention, SquaredReLU
from .registry import ModelFamily, register
from .transformer import TokenHead


@dataclass
class TaminexLayer:
    kind: str                         # "delta", "latent_attention" or "attention"
    heads: int
    dim: int
    vdim: int
    kv_heads: int = 0                 # delta (key heads) and attention
    conv: int = 0                     # delta: taps of the convolution
    scale: float = 1.0                # attention, latent_attention
    rot_dims: int = 0                 # attention
    rot_base: float = 10000.0
    kv_rank: int = 0                  # latent_attention
    kv_from: Optional[int] = None     # latent_attention: the layer whose latent rows it reads
    d_ff: int = 0                     # 0: no feed-forward

    @classmethod
    def from_dict(cls, d: dict) -> "TaminexLayer":
        kind, m, mlp = d["type"], d["mixer"], d.get("mlp")
        if mlp is not None and mlp.get("kind", "dense") != "dense":
            raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
        c = cls(kind=kind, heads=m["heads"], dim=m["dim"], vdim=m["vdim"], d_ff=mlp["ff"] if mlp else 0)
        if kind == "delta":
            c.kv_heads, c.conv = m["kv_heads"], m["conv"]
        elif kind == "attention":
            rot = m.get("rot") or {}
            c.kv_heads, c.scale = m["kv_heads"], float(m["scale"])
            c.rot_dims, c.rot_base = int(rot.get("dims", 0)), float(rot.get("base", c.rot_base))
            if c.rot_dims % 2 or c.rot_dims > c.dim:
                raise ValueError("rotated channels come in pairs inside the head")
        elif kind == "latent_attention":
            c.kv_rank, c.scale, c.kv_from = m["kv_rank"], float(m["scale"]), m.get("kv_from")
        else:
            raise ValueError(f"unsupported mixer type {kind!r}")
        if c.kv_heads and c.heads % c.kv_heads:
            raise ValueError("heads must be a multiple of kv_heads")
        return c

    def to_dict(self) -> dict:
        m = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}
        if self.kind == "delta":
            m.update(kv_heads=self.kv_heads, conv=self.conv)
        elif self.kind == "attention":
            m.update(kv_heads=self.kv_heads, scale=self.scale, rot={"dims": self.rot_dims, "base": self.rot_base})
        else:
            m.update(kv_rank=self.kv_rank, scale=self.scale)
            if self.kv_from is not None:
                m["kv_from"] = self.kv_from
        return {"type": self.kind, "mixer": m, "mlp": {"kind": "dense", "ff": self.d_ff} if self.d_ff else None}


@dataclass
class TaminexConfig:
    vocab_size: int
    d_model: int
    eps: float
    logit_scale: float
    logit_softcap: float                      # 0: no cap
    layers: list = field(default_factory=list)
    context_length: Optional[int] = None      # positions are unbounded; None = as long as the cache pool holds

    def __post_init__(self):
        for i, c in enumerate(self.layers):
            if c.kv_from is None:
                continue
            j = self.layers[c.kv_from] if 0 <= c.kv_from < i else None
            if j is None or j.kind != "latent_attention" or j.kv_from is not None or j.kv_rank != c.kv_rank:
                raise ValueError(f"layer {i}: kv_from must name an earlier latent layer with rows of its own, of the same rank")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    @classmethod
    def from_dict(cls, d: dict) -> "TaminexConfig":
        return cls(vocab_size=d["vocab"], d_model=d["width"], eps=float(d["norm"]["eps"]),
                   logit_scale=float(d.get("logit_scale", 1.0)), logit_softcap=float(d.get("logit_softcap") or 0.0),
                   layers=[TaminexLayer.from_dict(x) for x in d["layers"]], context_length=d.get("context_length"))

    def to_dict(self) -> dict:
        out = {"architecture": "Taminex", "vocab": self.vocab_size, "width": self.d_model, "norm": {"eps": self.eps},
               "logit_scale": self.logit_scale, "logit_softcap": self.logit_softcap,
               "layers": [x.to_dict() for x in self.layers]}
        if self.context_length is not None:
            out["context_length"] = self.context_length
        return out


class TaminexBlock(nn.Module):
    def __init__(self, p: Params, cfg: TaminexConfig, c: TaminexLayer, earlier: list):
        super().__init__()
        d, m = cfg.d_model, p.at("mix.")
        if c.kind == "delta":
            self.mixer = GatedDeltaRule(m, d, c.heads, c.kv_heads, c.dim, c.vdim, c.conv, cfg.eps)
        elif c.kind == "attention":
            self.mixer = SinkAttention(m, d, c.heads, c.kv_heads, c.dim, c.vdim, c.scale, c.rot_dims, c.rot_base, cfg.eps)
        else:
            source = earlier[c.kv_from].mixer if c.kv_from is not None else None
            self.mixer = LatentAttention(m, d, c.heads, c.dim, c.vdim, c.kv_rank, c.scale, cfg.eps, source)
        self.sublayers = [(self.mixer, p.f32("norm1", (d,)))]          # (sublayer, norm of its output)
        if c.d_ff:
            self.mlp = SquaredReLU(p.at("mlp."), d, c.d_ff)
            self.sublayers.append((self.mlp, p.f32("norm2", (d,))))


class TaminexLM(TokenHead, nn.Module):
    """``model(input_ids)`` -> final-norm hidden states [T, d]; the head is the one all models of the engine share, with
    the embedding as its matrix and a scale and soft cap behind it."""

    # what the engine needs to know (engine/model_runner.py, engine/llm_engine.py)
    mixed_batches = True        # portions of prompts and decoded tokens share a step
    splits_steps = True         # ... and the single tokens of such a step run on the decode kernels

    def __init__(self, cfg: TaminexConfig, weights: dict, device, dtype=torch.float32):
        super().__init__()
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        self.recurrent_state = any(c.kind == "delta" for c in cfg.layers)     # per-sequence state slots; no prefix reuse
        p = Params(weights, self.device, dtype)
        self.embed = p.lin("embed", (cfg.vocab_size, cfg.d_model))
        self.layers = nn.ModuleList()
        for i, c in enumerate(cfg.layers):
            self.layers.append(TaminexBlock(p.at(f"l{i}."), cfg, c, list(self.layers)))
        self.final_norm = p.f32("final.norm", (cfg.d_model,))
        self.w_head, self.b_head = self.embed, None
        self.sublayers = [s for layer in self.layers for s in layer.sublayers]

    def cache_owners(self):
        """Modules with pools to allocate, layer by layer."""
        return [layer.mixer for layer in self.layers]

    def prefill_tile_rows(self) -> int:
        return 0        # the layers ask for the tile lists they need (Portions.plan)

    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor | None = None) -> torch.Tensor:
        ctx, cfg = get_context(), self.cfg
        if positions is None:
            positions = ctx.positions if ctx.positions is not None else ctx.context_lens - 1
        x = torch.empty(input_ids.shape[0], cfg.d_model, dtype=torch.float32, device=input_ids.device)
        final = lambda i: self.final_norm if i == len(self.sublayers) else None
        h = ops.residual_norm(x, cfg.eps, self.dtype, tokens=input_ids, embed=self.embed, final_w=final(0))
        for i, (sub, norm) in enumerate(self.sublayers, 1):
            h = ops.residual_norm(x, cfg.eps, self.dtype, y=sub(h, ctx, positions), norm_w=norm, final_w=final(i))
        return h

    # ------------------------------------------------------------------ head
    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return ops.softcap_logits(self.logits_f32(hidden), self.cfg.logit_scale, self.cfg.logit_softcap)

    def greedy_tokens(self, hidden: torch.Tensor, out: torch.Tensor | None = None) -> torch.Tensor:
        if self.cfg.logit_scale > 0:        # scale and cap are increasing: the largest logit stays the largest
            return super().greedy_tokens(hidden, out)
        return ops.sample(self.compute_logits(hidden), None, 0, 0, out=out)


@torch.no_grad()
def init_weights(cfg: TaminexConfig, seed: int = 0, dtype=torch.float32) -> dict[str, torch.Tensor]:
    """Random parameters of the family's shapes under its checkpoint names (weights to run or test with, not a published
    initialisation): matrices N(0, 1/fan_in), decays from slow to fast, sinks around zero."""
    g = torch.Generator().manual_seed(seed)
    d = cfg.d_model
    w: dict[str, torch.Tensor] = {}

    def lin(name, n, k):
        w[name] = (torch.randn(n, k, generator=g) * k ** -0.5).to(dtype)

    def vec(name, n, mean, std):
        w[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    w["embed"] = torch.randn(cfg.vocab_size, d, generator=g).to(dtype)
    for i, c in enumerate(cfg.layers):
        p, m = f"l{i}.", f"l{i}.mix."
        if c.kind == "delta":
            for name, n in (("q", c.kv_heads * c.dim), ("k", c.kv_heads * c.dim), ("v", c.heads * c.vdim)):
                lin(m + name, n, d)
                w[m + name + ".conv"] = (torch.randn(n, c.conv, generator=g) * c.conv ** -0.5).to(dtype)
            lin(m + "b", c.heads, d)
            lin(m + "a", c.heads, d)
            vec(m + "A_log", c.heads, -1.5, 1.5)
            vec(m + "dt_bias", c.heads, -1.5, 1.0)
            vec(m + "norm", c.vdim, 1.0, 0.1)
            lin(m + "g", c.heads * c.vdim, d)
        elif c.kind == "attention":
            for name, n in (("q", c.heads * c.dim), ("k", c.kv_heads * c.dim), ("v", c.kv_heads * c.vdim)):
                lin(m + name, n, d)
                vec(m + name + ".b", n, 0.0, 0.3)
            vec(m + "q.norm", c.dim, 1.0, 0.2)
            vec(m + "k.norm", c.dim, 1.0, 0.2)
            vec(m + "sink", c.heads, 0.5, 1.0)
        else:
            lin(m + "q", c.heads * c.dim, d)
            if c.kv_from is None:
                lin(m + "dkv", c.kv_rank, d)
                vec(m + "dkv.norm", c.kv_rank, 1.0, 0.2)
            lin(m + "uk", c.heads * c.dim, c.kv_rank)
            lin(m + "uv", c.heads * c.vdim, c.kv_rank)
            lin(m + "g", c.heads * c.vdim, d)
        lin(m + "o", d, c.heads * c.vdim)
        vec(p + "norm1", d, 0.7, 0.1)
        if c.d_ff:
            lin(p + "mlp.up", c.d_ff, d)
            lin(p + "mlp.down", d, c.d_ff)
            vec(p + "norm2", d, 0.7, 0.1)
    vec("final.norm", d, 1.0, 0.1)
    return w


register(ModelFamily("Taminex", TaminexConfig, TaminexLM, init_weights))
