"""Small Taminex configurations and weights for the tests (sizes of their own, random weights, and weights shaped so that
a far key shows)."""
import torch

from oracle import taminex as orc


def _layer(kind, mixer, ff):
    return {"type": kind, "mixer": mixer, "mlp": None if ff is None else {"kind": "dense", "ff": ff}}


def delta(heads=4, kv_heads=2, dim=32, vdim=48, conv=4, ff=72):
    return _layer("delta", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, conv=conv), ff)


def latent(heads=3, dim=32, vdim=48, kv_rank=80, scale=None, kv_from=None, ff=72):
    m = dict(heads=heads, dim=dim, vdim=vdim, kv_rank=kv_rank, scale=dim ** -0.5 if scale is None else scale)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return _layer("latent_attention", m, ff)


def attention(heads=4, kv_heads=2, dim=48, vdim=32, scale=None, dims=16, base=10000.0, ff=72):
    return _layer("attention", dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim,
                                    scale=dim ** -0.5 if scale is None else scale, rot=dict(dims=dims, base=base)), ff)


def config(layers=None, vocab=131, width=112, eps=1e-5, scale=0.7, cap=12.0):
    layers = layers if layers is not None else [
        latent(), delta(), attention(), latent(heads=5, dim=16, vdim=16, kv_from=0, ff=None), delta(heads=3, kv_heads=3, dim=16,
                                                                                                vdim=32, conv=3, ff=None)]
    return {"architecture": "Taminex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": scale,
            "logit_softcap": cap, "layers": layers}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    from llm_from_scratch_b200.model import init_weights
    return {k: v.to(dtype) for k, v in init_weights(cfg, seed).items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def reference(cfg, w, ids):
    return orc.forward(cfg, w, ids)


MARK, SEEK = 7, 8      # the token that marked_keys marks, and the token that looks for it


def marked_keys(cfg, w, strength=30.0):
    """The same weights, but one channel of every attention key reads only an embedding channel that is large for token
    MARK alone, and the same channel of every query one that is large for token SEEK alone: the score of a SEEK query at a
    MARK key stands out by far, so that whether the query sees the key decides its logits.  In rotated heads the channel
    is the first that passes unrotated; sinks are low."""
    w = {k: v.clone() for k, v in w.items()}
    w["embed"][:, :2] = 0
    w["embed"][MARK, 0] = w["embed"][SEEK, 1] = 8.0
    for i, lay in enumerate(cfg["layers"]):
        c, p = lay["mixer"], f"l{i}.mix."
        for name in ("norm1", "norm2"):           # the marking channels of the residual stay clean
            if f"l{i}.{name}" in w:
                w[f"l{i}.{name}"][:2] = 0.0
        if lay["type"] == "delta":
            continue
        at = c["rot"]["dims"] if lay["type"] == "attention" else 0
        q_rows = torch.arange(c["heads"]) * c["dim"] + at
        w[p + "q"][q_rows] = 0
        w[p + "q"][q_rows, 1] = strength
        if lay["type"] == "attention":
            k_rows = torch.arange(c["kv_heads"]) * c["dim"] + at
            w[p + "k"][k_rows] = 0
            w[p + "k"][k_rows, 0] = strength
            for name, rows in (("q.b", q_rows), ("k.b", k_rows)):
                w[p + name][rows] = 0
            w[p + "sink"][:] = -1.0
        else:
            if p + "dkv" in w:
                w[p + "dkv"][0] = 0
                w[p + "dkv"][0, 0] = strength
                w[p + "dkv.norm"][:] = 1.0
            w[p + "uk"][q_rows] = 0
            w[p + "uk"][q_rows, 0] = 2.0
    return w


def plain_tokens(cfg, n, seed):
    """Tokens without MARK and SEEK."""
    return [t if t not in (MARK, SEEK) else SEEK + 1 for t in tokens(cfg, n, seed)]
