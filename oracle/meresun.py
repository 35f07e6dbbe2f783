"""CPU restatement of the Meresun decoder, one function per mechanism (test oracle).

A plain implementation that processes one sequence at a time from its first token, with no cache and no batching:
attention looks at every earlier position of the sequence through an explicit mask, experts are loops over tokens.
``dtype`` is the arithmetic type (float64 by default, so that the comparison measures the product path's rounding only).
It shares no code with ``llm_from_scratch_b200``.

Notation: n tokens, width d, H heads, r latent rank, i a query position, j a key position.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------ norms
def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return rms(x, eps) * w


def group_norm(x, w, groups, eps):
    """Every one of ``groups`` consecutive equal parts by its own root mean square, then the weight of the whole."""
    parts = x.view(*x.shape[:-1], groups, x.shape[-1] // groups)
    return rms(parts, eps).reshape(x.shape) * w


# --------------------------------------------------------------------------------------------- rotation
def rotary_frequencies(dims, base, scaling=None):
    """(f_i for i < dims / 2, factor of cos and sin).  With ``scaling`` the slow pairs turn ``factor`` times slower, the fast
    ones as they are, those between on a linear ramp over i; the ends of the ramp are the pairs that turn ``fast`` and
    ``slow`` times within ``original`` positions."""
    i = torch.arange(dims // 2, dtype=torch.float64)
    f = float(base) ** (-2 * i / dims)
    if scaling is None:
        return f, 1.0
    pair = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo, hi = max(math.floor(pair(scaling["fast"])), 0), min(math.ceil(pair(scaling["slow"])), dims - 1)
    ramp = ((i - lo) / max(hi - lo, 0.001)).clamp(0, 1)
    return f / scaling["factor"] * ramp + f * (1 - ramp), 0.1 * math.log(scaling["factor"]) + 1


def rotate_pairs(x, dims, base, scaling=None, first=0):
    """Rotary positions first, first + 1, ... on the first ``dims`` channels of x [n, heads, d], channel 2i with 2i + 1."""
    f, size = rotary_frequencies(dims, base, scaling)
    y = x.clone()
    for i in range(dims // 2):
        a = torch.arange(first, first + x.shape[0], dtype=torch.float64) * f[i]
        cos, sin = (size * torch.cos(a)).to(x.dtype)[:, None], (size * torch.sin(a)).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * cos - v * sin
        y[..., 2 * i + 1] = v * cos + u * sin
    return y


# -------------------------------------------------------------------------------------------- attention
def window_mask(nq, nk, window, first):
    """True where the query at position first + i does not see key j: later ones, and with ``window`` > 0 those
    ``window`` or more positions back."""
    i, j = torch.arange(first, first + nq)[:, None], torch.arange(nk)[None, :]
    hidden = j > i
    return hidden | (i - j >= window) if window else hidden


def windowed_attention(q, k, v, scale, sink=None, window=0, first=0):
    """Heads [nq, H, dv] of queries at positions first .. first + nq - 1 over keys 0 .. nk - 1.  ``sink`` [H] adds
    exp(sink) to the denominator only."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    s = s.masked_fill(window_mask(q.shape[0], k.shape[0], window, first)[None], -math.inf)
    if sink is not None:
        s = torch.cat([s, sink.view(-1, 1, 1).expand(-1, q.shape[0], 1)], -1)
    return torch.einsum("hij,jhd->ihd", torch.softmax(s, -1)[..., :k.shape[0]], v)


def latent_rows(h, w, c, eps):
    """(latents [n, r], rotated key part [n, rot_dim] shared by the heads)."""
    y = h @ w["dkv"].T
    rot = c["rot"]
    pe = rotate_pairs(y[:, None, c["kv_rank"]:], rot["dims"], rot["base"], rot.get("scaling"))[:, 0]
    return rms_norm(y[:, :c["kv_rank"]], w["dkv.norm"], eps), pe


def latent_queries(h, w, c, eps):
    n, H, dim, rot = h.shape[0], c["heads"], c["dim"], c["rot"]
    q = (rms_norm(h @ w["dq"].T, w["dq.norm"], eps) @ w["uq"].T).view(n, H, dim + c["rot_dim"])
    return torch.cat([q[..., :dim], rotate_pairs(q[..., dim:], rot["dims"], rot["base"], rot.get("scaling"))], -1)


def latent_mixer(h, w, c, eps):
    n, H = h.shape[0], c["heads"]
    latent, pe = latent_rows(h, w, c, eps)
    k = torch.cat([(latent @ w["uk"].T).view(n, H, c["dim"]), pe[:, None].expand(n, H, c["rot_dim"])], -1)
    v = (latent @ w["uv"].T).view(n, H, c["vdim"])
    window = (c.get("mask") or {}).get("size") or 0
    return windowed_attention(latent_queries(h, w, c, eps), k, v, c["scale"], w["sink"], window).reshape(n, -1) @ w["o"].T


# ----------------------------------------------------------------------------------------- feed-forwards
def poly_norm(z, a, eps):
    """a0 N(z) + a1 N(z^2) + a2 N(z^3) + a3, N over the token's vector."""
    return a[0] * rms(z, eps) + a[1] * rms(z ** 2, eps) + a[2] * rms(z ** 3, eps) + a[3]


def dense_mlp(h, w, eps):
    return poly_norm(h @ w["up"].T, w["act"], eps) @ w["down"].T


def clamped_glu(gate, up, limit, slope=1.702):
    g, u = gate.clamp(max=limit), up.clamp(-limit, limit)
    return g * torch.sigmoid(slope * g) * (u + 1)


def route(h, w_router, correction, groups, keep, top):
    """Per token the chosen experts (a set, ascending), their weights, and the margin of the choice: how far the last kept
    group is from the next, and the last chosen expert from the next one allowed, whichever is closer."""
    s = torch.sigmoid(h @ w_router.T)
    out = []
    for t in range(h.shape[0]):
        choice = [float(s[t, e] + correction[e]) for e in range(s.shape[1])]
        size = len(choice) // groups
        score = [sum(sorted(choice[g * size:(g + 1) * size])[-2:]) for g in range(groups)]
        best = sorted(range(groups), key=lambda g: -score[g])[:keep]
        allowed = [e for e in range(len(choice)) if e // size in best]
        ranked = sorted(allowed, key=lambda e: -choice[e])
        chosen = sorted(ranked[:top])
        gaps = [choice[ranked[top - 1]] - choice[ranked[top]]] if top < len(ranked) else []
        if keep < groups:
            order = sorted(score, reverse=True)
            gaps.append(order[keep - 1] - order[keep])
        out.append((chosen, s[t, chosen] / (s[t, chosen].sum() + 1e-20), min(gaps, default=math.inf)))
    return out


def moe_mlp(h, w, c, margins=None):
    r, rows = c["router"], []
    g = r.get("groups") or {"count": 1, "keep": 1}
    choices = route(h, w["router"], w["correction"], g["count"], g["keep"], r["top"])
    if margins is not None:
        margins.append([m for _, _, m in choices])
    for x, (chosen, weights, _) in zip(h, choices):
        y = torch.zeros_like(x)
        for e, p in zip(chosen, weights):
            act = clamped_glu(w[f"e{e}.gate"] @ x, w[f"e{e}.up"] @ x, c["expert"]["limit"])
            y = y + p * (w[f"e{e}.down"] @ act)
        rows.append(y)
    return torch.stack(rows)


# ------------------------------------------------------------------------------------ around the sublayers
def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def residual_gate(h, w, b):
    return torch.sigmoid(h @ w.T + b)


def token_input(x, e, w, eps):
    """x + norm(proj (gelu(gate x) * e)), e [n, dim] this layer's part of the tokens' side rows."""
    y = (gelu_tanh(x @ w["side.gate"].T) * e) @ w["side.proj"].T
    return x + rms_norm(y, w["side.norm"], eps)


def layer_runs(config):
    """(layer, an added embedding output comes first) in the order in which the layers run."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for k in range(loop["times"]):
        runs += [(i, k > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


# --------------------------------------------------------------------------------------- the model
def _sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, collect=None, margins=None):
    """Logits [n, vocab] of one sequence; ``collect`` (a list) receives the residual after every layer run, ``margins`` the
    margins of every routing, per token."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps, groups = config["norm"]["eps"], config["norm"].get("groups", 1)
    ids = torch.as_tensor(tokens, dtype=torch.long)
    start = w["embed"][ids] * config["embedding"]["scale"]
    side, dim = w["side.embed"][ids], config["token_side"]["dim"]
    x = start
    for i, again in layer_runs(config):
        layer, lw = config["layers"][i], _sub(w, f"l{i}.")
        if again:
            x = x + start
        h = group_norm(x, lw["norm1"], groups, eps)
        y = latent_mixer(h, _sub(lw, "mix."), layer["mixer"], eps) * residual_gate(h, lw["rg1"], lw["rg1.b"])
        mlp = layer.get("mlp")
        if mlp is not None:
            m = _sub(lw, "mlp.")
            f = dense_mlp(h, m, eps) if mlp["kind"] == "dense" else moe_mlp(h, m, mlp, margins)
            y = y + f * residual_gate(h, lw["rg2"], lw["rg2.b"])
        x = token_input(x + y, side[:, i * dim:(i + 1) * dim], lw, eps)
        if collect is not None:
            collect.append(x)
    return group_norm(x, w["final.norm"], groups, eps) @ w["head"].T


def greedy(config, weights, prompt, n_new, dtype=torch.float64):
    """(generated ids, margin between the two largest logits at every generated position)."""
    ids, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(config, weights, ids, dtype)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margins
