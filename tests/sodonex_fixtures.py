"""Small Sodonex configurations and weights for the tests (sizes of their own, random weights whose experts are chosen by clear
margins, and weights shaped so that a marked key shows)."""
import torch

MARK, SEEK = 7, 8      # the token that marked_keys marks, and the token that looks for it


def moe(ff=40, experts=7, top=3):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}


def layer(mlp="default", heads=6, kv_heads=2, dim=24, conv=4, chunk=50, rot_dims=8, base=1000.0, scale=None):
    m = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=dim, conv=conv, scale=1.3 * dim ** -0.5 if scale is None else scale,
             rot=dict(dims=rot_dims, base=base), mask={"size": chunk} if chunk else None)
    return {"type": "attention", "mixer": m, "mlp": moe() if mlp == "default" else mlp}


def config(layers=None, vocab=131, width=120, eps=1e-5, embed_scale=1.7, mult=0.4):
    layers = layers if layers is not None else [layer(), layer(heads=3, kv_heads=3, conv=2, chunk=37), layer(None, rot_dims=24, chunk=64),
                                                layer(moe(24, 9, 1), heads=4, kv_heads=1, dim=32, conv=3, chunk=16)]
    return {"architecture": "Sodonex", "vocab": vocab, "width": width, "norm": {"eps": eps}, "embedding": {"scale": embed_scale},
            "residual_mult": mult, "layers": layers}


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def _keep_clean(cfg, w, channels):
    """No sublayer writes these channels of the residual."""
    for name in w:
        if name.endswith(("mix.o", "mix.o.b", ".down")):
            w[name][channels] = 0


def weights(cfg, seed=0, dtype=torch.bfloat16):
    """Random weights; the experts' logits come from channels that hold a permutation of 0, 0.7, 1.4, ... per token, plus a
    little of everything else: their order does not hang on a rounding, their softmax on the whole input."""
    from llm_from_scratch_b200.model import init_weights
    w, g = init_weights(cfg, seed), torch.Generator().manual_seed(seed + 1)
    E = max((lay["mlp"]["router"]["experts"] for lay in cfg["layers"] if lay["mlp"]), default=0)
    first = 2                                            # channels 0 and 1 are marked_keys'
    assert first + E <= cfg["width"]
    _keep_clean(cfg, w, slice(0, first + E))
    w["embed"][:, first:first + E] = torch.rand(cfg["vocab"], E, generator=g).argsort(-1) * 0.7 / cfg["embedding"]["scale"]
    for i, lay in enumerate(cfg["layers"]):
        if lay["mlp"]:
            n = lay["mlp"]["router"]["experts"]
            r = w[f"l{i}.mlp.router"]
            r *= 0.04 / max(cfg["embedding"]["scale"], 1.0)
            r[:, first:first + E] = 0
            r[torch.arange(n), first + torch.randperm(E, generator=g)[:n]] = 1.0
            w[f"l{i}.mlp.router.b"] *= 0.1
    return {k: v.to(dtype) for k, v in w.items()}


def marked_keys(cfg, w, strength=4.0):
    """The same weights, but the last (unrotated) channel of every key reads only a channel that is large for token MARK alone,
    and that of every query one that is large for token SEEK alone, both without their neighbours: the score of a SEEK query at a
    MARK key stands out by far while other weights are small, so that whether the query sees the key decides its logits."""
    w = {k: v.clone() for k, v in w.items()}
    _keep_clean(cfg, w, slice(0, 2))
    w["embed"][:, :2] = 0
    w["embed"][MARK, 0] = w["embed"][SEEK, 1] = 8.0
    for i, lay in enumerate(cfg["layers"]):
        c, p = lay["mixer"], f"l{i}.mix."
        assert c["rot"]["dims"] < c["dim"]
        w[f"l{i}.shift"][:2] = 0
        for name, heads, channel in (("q", c["heads"], 1), ("k", c["kv_heads"], 0)):
            rows = torch.arange(heads) * c["dim"] + c["dim"] - 1
            w[p + name][rows] = 0
            w[p + name][rows, channel] = strength
            w[p + name + ".b"][rows] = 0
            w[p + name + ".conv"][rows] = 0
            w[p + name + ".conv"][rows, -1] = 1.0
            w[p + name + ".norm"][rows] = 2.0
        w[p + "pb"][:] = -5.0
    return w


def plain_tokens(cfg, n, seed):
    """Tokens without MARK and SEEK."""
    return [t if t not in (MARK, SEEK) else SEEK + 1 for t in tokens(cfg, n, seed)]
