"""CPU restatement of the Nabalix decoder, one function per mechanism (test oracle).

A plain implementation that processes one sequence at a time from its first token, with no cache and no
batching: attention looks at every earlier position of the sequence through an explicit mask, the recurrence
is a loop over tokens.  ``dtype`` is the arithmetic type (float64 by default, so that the comparison measures
the product path's rounding only).  It shares no code with ``llm_from_scratch_b200``.

Notation: n tokens, width d, streams s, H query heads over G key heads, i a query position, j a key position.
"""
from __future__ import annotations

import math

import torch


# ------------------------------------------------------------------------------------------------ norms
def rms(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def norm_one_plus(x, w, eps):
    return rms(x, eps) * (1 + w)


def norm_plain(x, w, eps):
    return rms(x, eps) * w


# ------------------------------------------------------------------------------- hyper-connections
def streams_read(X, w_in):
    """Sublayer input u[n, d] = sum_s w_in[s] X[s, n, d]."""
    return torch.einsum("s,snd->nd", w_in, X)


def streams_write(X, y, mix, w_out):
    """X'[t] = sum_s mix[s, t] X[s] + w_out[t] y."""
    return torch.einsum("st,snd->tnd", mix, X) + w_out[:, None, None] * y[None]


# --------------------------------------------------------------------------------------- attention
def distance_bias(r1, r2, dist):
    """r1[h] ln(1 + r2[h] dist) for a matrix of distances: [H, *dist.shape]."""
    shape = (-1,) + (1,) * dist.dim()
    return r1.view(shape) * torch.log(1 + r2.view(shape) * dist[None].to(r1.dtype))


def attention_weights(q, k, scale, softcap, r1, r2, talk, window, first=0):
    """[H, nq, nk] softmax weights for queries at positions first .. first + nq - 1 over keys 0 .. nk - 1.

    Per head: scale, soft cap, distance bias; the heads are then mixed by ``talk``; positions outside
    0 <= i - j < window carry no weight."""
    H, G = q.shape[1], k.shape[1]
    kh = k[:, torch.arange(H) // (H // G)]                          # the key head of every query head
    s = torch.einsum("ihd,jhd->hij", q, kh) * scale
    s = softcap * torch.tanh(s / softcap)
    i = torch.arange(first, first + q.shape[0])[:, None]
    j = torch.arange(k.shape[0])[None, :]
    dist = i - j
    s = s - distance_bias(r1, r2, dist.clamp(min=0))
    s = torch.einsum("hg,gij->hij", talk, s)
    seen = dist >= 0
    if window:
        seen = seen & (dist < window)
    s = s.masked_fill(~seen[None], -math.inf)
    return torch.softmax(s, -1)


def attention(q, k, v, scale, softcap, r1, r2, talk, window, first=0):
    """Heads [nq, H, dv]."""
    H, G = q.shape[1], v.shape[1]
    p = attention_weights(q, k, scale, softcap, r1, r2, talk, window, first)
    return torch.einsum("hij,jhd->ihd", p, v[:, torch.arange(H) // (H // G)])


def left_mixer(h, w, c):
    """Gated talking-heads attention of one whole sequence h [n, d]."""
    n, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = (h @ w["q"].T).view(n, H, c["dim"])
    k = (h @ w["k"].T).view(n, G, c["dim"])
    v = (h @ w["v"].T).view(n, G, c["vdim"])
    o = attention(q, k, v, c["scale"], c["softcap"], w["r1"], w["r2"], w["talk"], c["mask"]["size"])
    o = o.reshape(n, -1) * torch.sigmoid(h @ w["g"].T)
    return o @ w["o"].T


# -------------------------------------------------------------------------------------- recurrence
def forget_gate(z, bias, lower):
    """f = lower + (1 - lower) sigmoid(z + bias)."""
    return lower + (1 - lower) * torch.sigmoid(z + bias)


def gated_recurrence(q, f, v, state=None):
    """S <- diag(f) S + (1 - f) v^T, o = S^T q, token by token.  q, f [n, H, dk], v [n, H, dv];
    returns (o [n, H, dv], final state [H, dk, dv])."""
    n, H, dk = q.shape
    S = torch.zeros(H, dk, v.shape[2], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        S = f[t][:, :, None] * S + (1 - f[t])[:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def silu(x):
    return x * torch.sigmoid(x)


def right_mixer(h, w, c, eps):
    n, H, dk, dv = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = silu(h @ w["q"].T).view(n, H, dk)
    f = forget_gate(h @ w["f"].T, w["f.b"], w["lower"]).view(n, H, dk)
    v = (h @ w["v"].T).view(n, H, dv)
    o, _ = gated_recurrence(q, f, v)
    return norm_plain(o, w["norm"], eps).reshape(n, H * dv) @ w["o"].T


def parallel_join(left, right, w_left, w_right, eps):
    return (norm_plain(left, w_left, eps) + norm_plain(right, w_right, eps)) / 2


# ------------------------------------------------------------------------------------ feed-forward
def clamped_glu(g, u, limit):
    """min(g, limit) gated by its own sigmoid at slope 1.702, times clamp(u) + 1."""
    g = g.clamp(max=limit)
    u = u.clamp(-limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


# --------------------------------------------------------------------------------------- the model
def _sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, collect=None):
    """Logits [n, vocab] of one sequence; ``collect`` (a list) receives the sum of the streams after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    X = x[None].repeat(config["streams"], 1, 1)
    for i, layer in enumerate(config["layers"]):
        lw = _sub(w, f"l{i}.")

        def sublayer(X, q, fn):
            hc = _sub(lw, f"hc{q}.")
            u = streams_read(X, hc["in"])
            y = fn(norm_one_plus(u, lw[f"norm{q}"], eps)) * lw[f"ls{q}"]
            return streams_write(X, y, hc["mix"], hc["out"])

        def mixer(h):
            left = left_mixer(h, _sub(lw, "mix.left."), layer["mixer"]["left"])
            right = right_mixer(h, _sub(lw, "mix.right."), layer["mixer"]["right"], eps)
            return parallel_join(left, right, lw["mix.left.out"], lw["mix.right.out"], eps)

        X = sublayer(X, 1, mixer)
        if layer.get("mlp") is not None:
            m = _sub(lw, "mlp.")
            X = sublayer(X, 2, lambda h: clamped_glu(h @ m["gate"].T, h @ m["up"].T, layer["mlp"]["limit"]) @ m["down"].T)
        if collect is not None:
            collect.append(X.sum(0))
    return norm_one_plus(X.sum(0), w["final.norm"], eps) @ w["head"].T


def greedy(config, weights, prompt, n_new, dtype=torch.float64):
    """(generated ids, margin between the two largest logits at every generated position)."""
    ids, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(config, weights, ids, dtype)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margins
