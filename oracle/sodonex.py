"""CPU restatement of the Sodonex decoder, one function per mechanism (test oracle).

A plain implementation that processes one sequence at a time from its first token, with no cache and no batching: the shift and
the convolution are loops over tokens, attention looks at every earlier position through an explicit mask, every token runs its
experts one by one.  ``dtype`` is the arithmetic type (float64 by default, so that the comparison measures the product path's
rounding only).  It shares no code with ``llm_from_scratch_b200``.

Notation: n tokens, width d, H query heads over G key heads of D channels, i a query position, j a key position.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------ norms
def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gain_norm(x, g, eps):
    """RMS norm with one number for all channels."""
    return rms(x, eps) * g.reshape(())


def whole_norm(x, w, eps):
    """RMS norm over all channels of a projection, before it is cut into heads."""
    return rms(x, eps) * w


# ------------------------------------------------------------------------------------- what tokens carry over
def token_shift(x, s):
    """h_t = x_t + (x_{t-1} - x_t) s, with zeros before the first token."""
    rows = []
    for t in range(x.shape[0]):
        before = x[t - 1] if t else torch.zeros_like(x[0])
        rows.append(x[t] + (before - x[t]) * s)
    return torch.stack(rows)


def short_conv(u, taps):
    """y_t = sum_m taps[:, m] u_{t - (M - 1) + m} per channel, zeros before the first token."""
    n, M = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(n):
        for m in range(M):
            s = t - (M - 1) + m
            if s >= 0:
                y[t] += taps[:, m] * u[s]
    return y


# --------------------------------------------------------------------------------------------- attention
def rotate_half(x, dims, base, first=0):
    """Rotary positions on the first ``dims`` channels of x [n, heads, D], channel i paired with i + dims / 2."""
    n, half = x.shape[0], dims // 2
    y = x.clone()
    for i in range(half):
        a = torch.arange(first, first + n, dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
        cos, sin = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., i], x[..., i + half]
        y[..., i] = u * cos - v * sin
        y[..., i + half] = v * cos + u * sin
    return y


def chunk_mask(nq, nk, first, size):
    """True where a query at position first + i does not see key j: later keys, and keys of another chunk (size 0: no chunks)."""
    i, j = torch.arange(first, first + nq)[:, None], torch.arange(nk)[None, :]
    hidden = j > i
    return hidden | (i // size != j // size) if size else hidden


def sigmoid_attention(q, k, v, scale, bias, size=0, first=0):
    """Sums [nq, H, D] of the values under the weights sigmoid(scale q.k + bias[h]), which are not normalised; queries at
    positions first .. first + nq - 1 over keys 0 .. nk - 1."""
    H, G = q.shape[1], k.shape[1]
    of = torch.arange(H) // (H // G)
    z = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale + bias.view(H, 1, 1)
    p = torch.sigmoid(z).masked_fill(chunk_mask(q.shape[0], k.shape[0], first, size)[None], 0.0)
    return torch.einsum("hij,jhd->ihd", p, v[:, of])


def mixer(h, w, c, eps):
    n, H, G, D = h.shape[0], c["heads"], c["kv_heads"], c["dim"]
    q = short_conv(h @ w["q"].T + w["q.b"], w["q.conv"])
    k = short_conv(h @ w["k"].T + w["k.b"], w["k.conv"])
    v = k.view(n, G, D)
    q, k = whole_norm(q, w["q.norm"], eps).view(n, H, D), whole_norm(k, w["k.norm"], eps).view(n, G, D)
    q, k = (rotate_half(x, c["rot"]["dims"], c["rot"]["base"]) for x in (q, k))
    o = sigmoid_attention(q, k, v, c["scale"], w["pb"], (c.get("mask") or {}).get("size", 0))
    o = o * torch.sigmoid(h @ w["g"].T)[..., None]
    return o.reshape(n, H * D) @ w["o"].T + w["o.b"]


# ------------------------------------------------------------------------------------------ feed-forward
def route(h, router, bias, top):
    """Per token: (chosen experts, their weights, margin): the ``top`` largest logits, softmax over those alone.  ``margin`` is
    the distance between the last chosen logit and the first one left out."""
    z, out = h @ router.T + bias, []
    for row in z:
        ranked = sorted(range(len(row)), key=lambda e: -row[e].item())
        chosen = ranked[:top]
        margin = (row[ranked[top - 1]] - row[ranked[top]]).item() if top < len(ranked) else math.inf
        out.append((chosen, torch.softmax(row[chosen], -1), margin))
    return out


def experts(h, w, c, margins=None):
    choices, rows = route(h, w["router"], w["router.b"], c["router"]["top"]), []
    if margins is not None:
        margins.append([m for _, _, m in choices])
    for x, (chosen, weights, _) in zip(h, choices):
        y = torch.zeros_like(x)
        for e, p in zip(chosen, weights):
            y = y + p * (w[f"e{e}.down"] @ (w[f"e{e}.up"] @ x).clamp(min=0) ** 2)
        rows.append(y)
    return torch.stack(rows)


# --------------------------------------------------------------------------------------- the model
def _sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, collect=None, margins=None):
    """Logits [n, vocab] of one sequence; ``collect`` (a list) receives the residual after every layer, ``margins`` the margins
    of every routing, per token."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)] * config["embedding"]["scale"]
    for i, layer in enumerate(config["layers"]):
        lw = _sub(w, f"l{i}.")
        h = token_shift(x, lw["shift"])
        x = x + m * gain_norm(mixer(h, _sub(lw, "mix."), layer["mixer"], eps), lw["norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + m * gain_norm(experts(x, _sub(lw, "mlp."), layer["mlp"], margins), lw["norm2"], eps)
        if collect is not None:
            collect.append(x)
    return gain_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(config, weights, prompt, n_new, dtype=torch.float64):
    """(generated ids, margin between the two largest logits at every generated position)."""
    ids, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(config, weights, ids, dtype)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margins
