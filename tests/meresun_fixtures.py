"""Small Meresun configurations and weights for the tests (sizes of their own, random weights, and weights shaped so that a
marked key shows)."""
import torch

from oracle import meresun as orc

YARN = dict(factor=4.0, original=64, fast=8.0, slow=1.0)


def dense(ff=72):
    return {"kind": "dense", "ff": ff}


def moe(ff=40, experts=12, top=3, groups=(3, 2), limit=0.8):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit},
            "router": {"experts": experts, "top": top, "groups": {"count": groups[0], "keep": groups[1]}}}


def layer(mlp=None, heads=3, dim=24, rot_dim=8, vdim=32, q_rank=40, kv_rank=48, window=37, base=1000.0, scaling=YARN, scale=None):
    rot = dict(dims=rot_dim, base=base)
    if scaling:
        rot["scaling"] = scaling
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, rot=rot,
             scale=(dim + rot_dim) ** -0.5 if scale is None else scale, mask={"size": window} if window else None)
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def config(layers=None, vocab=131, width=120, eps=1e-5, groups=3, embed_scale=0.7, side=20, loop=(1, 3, 2)):
    layers = layers if layers is not None else [layer(dense()), layer(moe(), heads=5, window=50), layer(None, scaling=None),
                                                layer(moe(groups=(1, 1)), window=16, rot_dim=16)]
    out = {"architecture": "Meresun", "vocab": vocab, "width": width, "norm": {"eps": eps, "groups": groups},
           "embedding": {"scale": embed_scale}, "token_side": {"dim": side}, "layers": layers}
    if loop:
        out["loop"] = dict(zip(("start", "stop", "times"), loop))
    return out


def weights(cfg, seed=0, dtype=torch.bfloat16):
    from llm_from_scratch_b200.model import init_weights
    return {k: v.to(dtype) for k, v in init_weights(cfg, seed).items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


MARK, SEEK = 7, 8      # the token that marked_keys marks, and the token that looks for it


def marked_keys(cfg, w, strength=30.0):
    """The same weights, but one latent channel of every key reads only an embedding channel that is large for token MARK
    alone, and one channel of every query one that is large for token SEEK alone: the score of a SEEK query at a MARK key
    stands out by far, so that whether the query sees the key decides its logits.  Sinks are low."""
    w = {k: v.clone() for k, v in w.items()}
    w["embed"][:, :2] = 0
    w["embed"][MARK, 0] = w["embed"][SEEK, 1] = 8.0
    for i, lay in enumerate(cfg["layers"]):
        c, p = lay["mixer"], f"l{i}.mix."
        for name in [p + "o"] + [n for n in w if n.startswith(f"l{i}.mlp.") and n.endswith("down")]:
            w[name][:2] = 0                                  # the marking channels of the residual stay clean
        w[f"l{i}.side.norm"][:2] = 0
        w[p + "dq"][0], w[p + "dkv"][0] = 0, 0
        w[p + "dq"][0, 1] = w[p + "dkv"][0, 0] = strength
        w[p + "dq.norm"][0] = w[p + "dkv.norm"][0] = 1.0
        q_rows, k_rows = torch.arange(c["heads"]) * (c["dim"] + c["rot_dim"]), torch.arange(c["heads"]) * c["dim"]
        w[p + "uq"][q_rows], w[p + "uk"][k_rows] = 0, 0
        w[p + "uq"][q_rows, 0] = w[p + "uk"][k_rows, 0] = 2.0
        w[p + "sink"][:] = -1.0
    return w


def plain_tokens(cfg, n, seed):
    """Tokens without MARK and SEEK."""
    return [t if t not in (MARK, SEEK) else SEEK + 1 for t in tokens(cfg, n, seed)]


def reference(cfg, w, ids, dtype):
    """The restatement's logits, and which positions' expert choices are further from a tie than the rounding of ``dtype``
    can bring them: where a tie breaks the other way, the token has another expert and its logits are another function."""
    margins = []
    want = orc.forward(cfg, w, ids, margins=margins)
    keep = torch.ones(len(ids), dtype=torch.bool)
    for m in margins:
        keep &= torch.tensor(m) > (0.012 if dtype == torch.bfloat16 else 1e-5)
    assert keep.float().mean() > 0.25 or len(ids) < 30
    return want, keep


def error(got, want):
    """``engine_helpers.error`` over the settled positions of ``reference``."""
    from engine_helpers import error
    logits, keep = want
    return error(got[keep], logits[keep]) if keep.any() else 0.0
