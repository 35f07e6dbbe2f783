"""The Meresun decoder family: windowed latent attention (query latents, YaRN-rotated shared key part, sinks) beside a PolyNorm
feed-forward or a grouped mixture of clamped GLU experts, both on one grouped norm and behind element-wise gates, an input per
layer from a token table, and a range of layers that runs several times with the same weights.

The module only composes mechanisms of ``mixers`` and the shared head; caches, batching and sampling are the engine's.
Parameter names are those of the family's checkpoints (``l<i>.mix.dq`` and so on).  The residual, norms, angles, scores, router
and gates are fp32 in either compute dtype; matrix products and activations between them are in the compute dtype.
"""
from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch
from torch import nn

from .. import ops
from ..utils.context import get_context
from .mixers import GatedSublayers, GroupedMoE, Params, PolyNormMLP, RotaryLatentAttention, RunCache, TokenInput
from .registry import ModelFamily, register
from .transformer import TokenHead


@dataclass
class MeresunLayer:
    heads: int
    dim: int                          # unrotated query / key channels per head
    rot_dim: int                      # rotated ones; their key part is shared by the heads
    vdim: int
    q_rank: int
    kv_rank: int
    scale: float
    rot_dims: int                     # channels of the rotary part that turn
    rot_base: float
    scaling: Optional[ops.YarnScaling] = None
    window: int = 0                   # 0: no window
    d_ff: int = 0                     # of the dense feed-forward or of every expert; 0: no feed-forward
    experts: int = 0                  # 0: dense
    top: int = 0
    groups: int = 1
    keep: int = 1
    limit: float = 0.0

    @classmethod
    def from_dict(cls, d: dict) -> "MeresunLayer":
        if d["type"] != "latent_attention":
            raise ValueError(f"unsupported mixer type {d['type']!r}")
        m, mlp = d["mixer"], d.get("mlp")
        rot, mask = m.get("rot") or {}, m.get("mask") or {}
        scaling = rot.get("scaling")
        c = cls(heads=m["heads"], dim=m["dim"], rot_dim=m["rot_dim"], vdim=m["vdim"], q_rank=m["q_rank"], kv_rank=m["kv_rank"],
                scale=float(m["scale"]), rot_dims=int(rot.get("dims", m["rot_dim"])), rot_base=float(rot.get("base", 10000.0)),
                scaling=ops.YarnScaling(*(float(scaling[k]) for k in ("factor", "original", "fast", "slow"))) if scaling else None,
                window=int(mask.get("size") or 0))
        if c.rot_dims % 2 or c.rot_dims > c.rot_dim:
            raise ValueError("rotated channels come in pairs inside the rotary part")
        if mlp is None:
            return c
        if mlp["kind"] == "dense":
            c.d_ff = mlp["ff"]
        elif mlp["kind"] == "moe":
            router, expert = mlp["router"], mlp["expert"]
            groups = router.get("groups") or {"count": 1, "keep": 1}
            c.d_ff, c.limit, c.experts, c.top = expert["ff"], float(expert["limit"]), router["experts"], router["top"]
            c.groups, c.keep = groups["count"], groups["keep"]
            if c.experts % c.groups or not 0 < c.keep <= c.groups or not 0 < c.top <= c.keep * (c.experts // c.groups):
                raise ValueError("experts must form equal groups, and the kept ones hold the experts a token uses")
        else:
            raise ValueError(f"unsupported feed-forward kind {mlp['kind']!r}")
        return c

    def to_dict(self) -> dict:
        rot = {"dims": self.rot_dims, "base": self.rot_base}
        if self.scaling is not None:
            rot["scaling"] = {k: getattr(self.scaling, k) for k in ("factor", "original", "fast", "slow")}
        mixer = dict(heads=self.heads, dim=self.dim, rot_dim=self.rot_dim, vdim=self.vdim, q_rank=self.q_rank,
                     kv_rank=self.kv_rank, scale=self.scale, rot=rot, mask={"size": self.window} if self.window else None)
        mlp = None
        if self.experts:
            mlp = {"kind": "moe", "expert": {"ff": self.d_ff, "limit": self.limit},
                   "router": {"experts": self.experts, "top": self.top, "groups": {"count": self.groups, "keep": self.keep}}}
        elif self.d_ff:
            mlp = {"kind": "dense", "ff": self.d_ff}
        return {"type": "latent_attention", "mixer": mixer, "mlp": mlp}


@dataclass
class MeresunConfig:
    vocab_size: int
    d_model: int
    eps: float
    norm_groups: int
    embed_scale: float
    side_dim: int                             # channels of a layer's part of the token table
    layers: list = field(default_factory=list)
    loop: Optional[tuple] = None              # (start, stop, times)
    context_length: Optional[int] = None      # positions are unbounded; None = as long as the cache pool holds

    def __post_init__(self):
        if self.d_model % self.norm_groups:
            raise ValueError("the norm's groups must divide the width")
        if self.loop is not None:
            start, stop, times = self.loop
            if not 0 <= start < stop <= len(self.layers) or times < 1:
                raise ValueError("a loop runs a range of the layers at least once")

    @property
    def num_layers(self) -> int:
        return len(self.layers)

    def layer_runs(self) -> list[tuple[int, bool]]:
        """(layer, whether it begins a pass of the loop after the first) in the order in which layers run."""
        start, stop, times = self.loop or (0, 0, 1)
        runs = [(i, False) for i in range(start)]
        for k in range(times):
            runs += [(i, k > 0 and i == start) for i in range(start, stop)]
        return runs + [(i, False) for i in range(stop, len(self.layers))]

    @classmethod
    def from_dict(cls, d: dict) -> "MeresunConfig":
        loop = d.get("loop")
        return cls(vocab_size=d["vocab"], d_model=d["width"], eps=float(d["norm"]["eps"]),
                   norm_groups=int(d["norm"].get("groups") or 1), embed_scale=float((d.get("embedding") or {}).get("scale", 1.0)),
                   side_dim=d["token_side"]["dim"], layers=[MeresunLayer.from_dict(x) for x in d["layers"]],
                   loop=(loop["start"], loop["stop"], loop["times"]) if loop else None, context_length=d.get("context_length"))

    def to_dict(self) -> dict:
        out = {"architecture": "Meresun", "vocab": self.vocab_size, "width": self.d_model,
               "norm": {"eps": self.eps, "groups": self.norm_groups}, "embedding": {"scale": self.embed_scale},
               "token_side": {"dim": self.side_dim}, "layers": [x.to_dict() for x in self.layers]}
        if self.loop is not None:
            out["loop"] = dict(zip(("start", "stop", "times"), self.loop))
        if self.context_length is not None:
            out["context_length"] = self.context_length
        return out


class MeresunBlock(nn.Module):
    def __init__(self, p: Params, cfg: MeresunConfig, i: int, table: torch.Tensor):
        super().__init__()
        d, c, m = cfg.d_model, cfg.layers[i], p.at("mix.")
        rotation = ops.Rotation(c.rot_base, c.rot_dims, p.device, c.scaling)
        mixer = RotaryLatentAttention(m, d, c.heads, c.dim, c.rot_dim, c.vdim, c.q_rank, c.kv_rank, c.scale, rotation, c.window,
                                      cfg.eps)
        mlp = None
        if c.experts:
            mlp = GroupedMoE(p.at("mlp."), d, c.d_ff, c.experts, c.top, c.groups, c.keep, c.limit)
        elif c.d_ff:
            mlp = PolyNormMLP(p.at("mlp."), d, c.d_ff, cfg.eps)
        self.norm = p.f32("norm1", (d,))
        self.sublayers = GatedSublayers(p, d, mixer, mlp)
        self.side = TokenInput(p.at("side."), d, table, i * cfg.side_dim, cfg.side_dim)


class MeresunLM(TokenHead, nn.Module):
    """``model(input_ids)`` -> final-norm hidden states [T, d]; the head is the one all models of the engine share."""

    # what the engine needs to know (engine/model_runner.py, engine/llm_engine.py)
    recurrent_state = False
    mixed_batches = True        # portions of prompts and decoded tokens share a step
    splits_steps = True         # ... and the single tokens of such a step run on the decode kernels

    def __init__(self, cfg: MeresunConfig, weights: dict, device, dtype=torch.float32):
        super().__init__()
        self.cfg, self.dtype, self.device = cfg, dtype, torch.device(device)
        p = Params(weights, self.device, dtype)
        self.embed = p.lin("embed", (cfg.vocab_size, cfg.d_model))
        table = p.lin("side.embed", (cfg.vocab_size, cfg.num_layers * cfg.side_dim))
        self.layers = nn.ModuleList([MeresunBlock(p.at(f"l{i}."), cfg, i, table) for i in range(cfg.num_layers)])
        # (layer, its cache in this run, whether the embedding joins the residual before it)
        self.runs = [(self.layers[i], RunCache(self.layers[i].sublayers.mixer), again) for i, again in cfg.layer_runs()]
        self.final_norm = p.f32("final.norm", (cfg.d_model,))
        self.w_head, self.b_head = p.lin("head", (cfg.vocab_size, cfg.d_model)), None
        # steps of whole prompts can be captured: every layer's attention then takes its grid from a tile list
        self.captures_prompts = all(layer.sublayers.mixer.tile_rows(dtype) for layer in self.layers)
        self.attention_windows = sorted({c.window for c in cfg.layers if c.window})

    def cache_owners(self):
        """Objects with pools to allocate, run by run."""
        return [pools for _, pools, _ in self.runs]

    def prefill_tile_rows(self) -> int:
        return 0        # the layers ask for the tile lists they need (Portions.plan)

    def forward(self, input_ids: torch.Tensor, positions: torch.Tensor | None = None) -> torch.Tensor:
        ctx, cfg = get_context(), self.cfg
        if positions is None:
            positions = ctx.positions if ctx.positions is not None else ctx.context_lens - 1
        x = torch.empty(input_ids.shape[0], cfg.d_model, dtype=torch.float32, device=input_ids.device)
        embedding = dict(tokens=input_ids, embed=self.embed, embed_scale=cfg.embed_scale)
        step = dict(embedding, start=True)
        for layer, pools, again in self.runs:
            if again:
                step.update(embedding)
            h = ops.residual_group_norm(x, layer.norm, cfg.norm_groups, cfg.eps, self.dtype, **step)
            y = layer.side(layer.sublayers(h, x, ctx, positions, pools), input_ids)
            step = dict(y=y, y_norm_w=layer.side.norm)
        return ops.residual_group_norm(x, self.final_norm, cfg.norm_groups, cfg.eps, self.dtype, **step)

    def compute_logits(self, hidden: torch.Tensor) -> torch.Tensor:
        return self.logits_f32(hidden)


@torch.no_grad()
def init_weights(cfg: MeresunConfig, seed: int = 0, dtype=torch.float32) -> dict[str, torch.Tensor]:
    """Random parameters of the family's shapes under its checkpoint names (weights to run or test with, not a published
    initialisation): matrices N(0, 1/fan_in), gates around one half, corrections that move some choices, sinks around zero."""
    g = torch.Generator().manual_seed(seed)
    d = cfg.d_model
    w: dict[str, torch.Tensor] = {}

    def lin(name, n, k):
        w[name] = (torch.randn(n, k, generator=g) * k ** -0.5).to(dtype)

    def vec(name, n, mean, std):
        w[name] = (mean + std * torch.randn(n, generator=g)).to(dtype)

    w["embed"] = torch.randn(cfg.vocab_size, d, generator=g).to(dtype)
    w["side.embed"] = torch.randn(cfg.vocab_size, cfg.num_layers * cfg.side_dim, generator=g).to(dtype)
    for i, c in enumerate(cfg.layers):
        p, m = f"l{i}.", f"l{i}.mix."
        vec(p + "norm1", d, 1.0, 0.1)
        lin(m + "dq", c.q_rank, d)
        vec(m + "dq.norm", c.q_rank, 1.0, 0.2)
        lin(m + "uq", c.heads * (c.dim + c.rot_dim), c.q_rank)
        lin(m + "dkv", c.kv_rank + c.rot_dim, d)
        vec(m + "dkv.norm", c.kv_rank, 1.0, 0.2)
        lin(m + "uk", c.heads * c.dim, c.kv_rank)
        lin(m + "uv", c.heads * c.vdim, c.kv_rank)
        vec(m + "sink", c.heads, 0.5, 1.0)
        lin(m + "o", d, c.heads * c.vdim)
        for q in ("rg1", "rg2") if c.d_ff else ("rg1",):
            lin(p + q, d, d)
            vec(p + q + ".b", d, 0.0, 0.3)
        if c.experts:
            lin(p + "mlp.router", c.experts, d)
            vec(p + "mlp.correction", c.experts, 0.0, 0.3)
            for e in range(c.experts):
                lin(f"{p}mlp.e{e}.gate", c.d_ff, d)
                lin(f"{p}mlp.e{e}.up", c.d_ff, d)
                lin(f"{p}mlp.e{e}.down", d, c.d_ff)
        elif c.d_ff:
            lin(p + "mlp.up", c.d_ff, d)
            lin(p + "mlp.down", d, c.d_ff)
            w[p + "mlp.act"] = torch.tensor([0.6, 0.4, 0.2, 0.1]).to(dtype) + (0.1 * torch.randn(4, generator=g)).to(dtype)
        lin(p + "side.gate", cfg.side_dim, d)
        lin(p + "side.proj", d, cfg.side_dim)
        vec(p + "side.norm", d, 0.4, 0.1)
    vec("final.norm", d, 1.0, 0.1)
    lin("head", cfg.vocab_size, d)
    return w


register(ModelFamily("Meresun", MeresunConfig, MeresunLM, init_weights))
