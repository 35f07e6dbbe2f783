"""Small Nabalix configurations and weights for the tests (sizes of their own, random weights, and weights shaped so
that a far key, a window's edge or a lost state shows)."""
import torch

from oracle import nabalix as orc


def layer(heads=4, kv_heads=2, dim=32, vdim=48, window=40, scale=None, softcap=20.0, rec=(3, 16, 32), ff=80, limit=2.0):
    return {"type": "parallel",
            "mixer": {"left": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim,
                               "scale": dim ** -0.5 if scale is None else scale, "softcap": softcap,
                               "mask": {"size": window}},
                      "right": {"heads": rec[0], "dim": rec[1], "vdim": rec[2]}},
            "mlp": None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}}


def config(layers=None, vocab=131, width=112, streams=3, eps=1e-5):
    layers = layers if layers is not None else [
        layer(), layer(heads=6, kv_heads=6, dim=16, vdim=32, window=9, ff=None, rec=(2, 48, 16)),
        layer(heads=5, kv_heads=1, dim=64, vdim=16, window=130, softcap=6.0, rec=(1, 80, 64), limit=0.7)]
    return {"architecture": "Nabalix", "vocab": vocab, "width": width, "streams": streams, "norm": {"eps": eps},
            "layers": layers}


def weights(cfg, seed=0, dtype=torch.bfloat16):
    from llm_from_scratch_b200.model import init_weights
    return {k: v.to(dtype) for k, v in init_weights(cfg, seed).items()}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def reference(cfg, w, ids):
    return orc.forward(cfg, w, ids)


MARK, SEEK = 7, 8      # the token that marked_keys marks, and the token that looks for it


def marked_keys(cfg, w, strength=12.0):
    """The same weights, but every head's first key channel reads only an embedding channel that is large for token
    MARK alone, and every head's first query channel one that is large for token SEEK alone: the score of a SEEK
    query at a MARK key stands out by far, so that whether the query sees the key decides its logits."""
    w = {k: v.clone() for k, v in w.items()}
    w["embed"][:, :2] = 0
    w["embed"][MARK, 0] = w["embed"][SEEK, 1] = 8.0
    for i, lay in enumerate(cfg["layers"]):
        c = lay["mixer"]["left"]
        for name, heads, channel in (("q", c["heads"], 1), ("k", c["kv_heads"], 0)):
            m = w[f"l{i}.mix.left.{name}"]
            first = torch.arange(heads) * c["dim"]
            m[first] = 0
            m[first, channel] = strength
        for name in ("norm1", "ls1", "ls2"):      # the marking channels stay clean
            if f"l{i}.{name}" in w:
                w[f"l{i}.{name}"][:2] = 0.0
    return w


def plain_tokens(cfg, n, seed):
    """Tokens without MARK and SEEK."""
    return [t if t not in (MARK, SEEK) else SEEK + 1 for t in tokens(cfg, n, seed)]
