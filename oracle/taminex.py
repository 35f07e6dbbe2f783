"""CPU restatement of the Taminex decoder, one function per mechanism (test oracle).

A plain implementation that processes one sequence at a time from its first token, with no cache and no batching:
attention looks at every earlier position of the sequence through an explicit mask, the recurrence and the
convolution are loops over tokens.  ``dtype`` is the arithmetic type (float64 by default, so that the comparison
measures the product path's rounding only).  It shares no code with ``llm_from_scratch_b200``.

Notation: n tokens, width d, H query (or value) heads over G key heads, i a query position, j a key position.
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


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    """ln(1 + e^x), written so that neither tail overflows."""
    return x.clamp(min=0) + torch.log1p(torch.exp(-x.abs()))


# ------------------------------------------------------------------------------------- gated delta rule
def short_conv(x, taps):
    """y[t] = sum_m taps[:, m] x[t - (M - 1) + m] per channel, zeros before the first token."""
    n, M = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(n):
        for m in range(M):
            s = t - (M - 1) + m
            if s >= 0:
                y[t] += taps[:, m] * x[s]
    return y


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def log_decay(z, dt_bias, a_log):
    """ln g = -exp(A) softplus(z + bias)."""
    return -torch.exp(a_log) * softplus(z + dt_bias)


def delta_rule(q, k, v, beta, log_g, state=None):
    """Token by token, per value head h with key head h // (H / G):
    S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q.
    q, k [n, G, dk], v [n, H, dv], beta, log_g [n, H]; returns (o [n, H, dv], final state [H, dk, dv])."""
    n, H, G = v.shape[0], v.shape[1], k.shape[1]
    of = torch.arange(H) // (H // G)
    S = torch.zeros(H, k.shape[2], v.shape[2], dtype=v.dtype) if state is None else state.clone()
    out = []
    for t in range(n):
        kt, qt = k[t][of], q[t][of]
        S = torch.exp(log_g[t])[:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, kt))
        S = S + kt[:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, qt))
    return torch.stack(out), S


def delta_mixer(h, w, c, eps):
    n, H, G, dk, dv = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q, k, v = (silu(short_conv(h @ w[x].T, w[x + ".conv"])) for x in "qkv")
    q = unit(q.view(n, G, dk)) * dk ** -0.5
    k = unit(k.view(n, G, dk))
    beta = torch.sigmoid(h @ w["b"].T)
    o, _ = delta_rule(q, k, v.view(n, H, dv), beta, log_decay(h @ w["a"].T, w["dt_bias"], w["A_log"]))
    o = rms_norm(o, w["norm"], eps).reshape(n, H * dv) * silu(h @ w["g"].T)
    return o @ w["o"].T


# --------------------------------------------------------------------------------------------- attention
def causal_attention(q, k, v, scale, sink=None, first=0):
    """Heads [nq, H, dv] of queries at positions first .. first + nq - 1 over keys 0 .. nk - 1.  ``sink`` [H] adds
    exp(sink) to the denominator only."""
    H, G = q.shape[1], k.shape[1]
    of = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q, k[:, of]) * scale
    i = torch.arange(first, first + q.shape[0])[:, None]
    s = s.masked_fill((torch.arange(k.shape[0])[None, :] > i)[None], -math.inf)
    if sink is not None:
        s = torch.cat([s, sink.view(H, 1, 1).expand(H, q.shape[0], 1)], -1)
    p = torch.softmax(s, -1)[..., :k.shape[0]]
    return torch.einsum("hij,jhd->ihd", p, v[:, of])


def rotate_pairs(x, dims, base, first=0):
    """Rotary positions on the first ``dims`` channels of x [n, heads, d], channel 2i paired with 2i + 1."""
    n = x.shape[0]
    y = x.clone()
    for i in range(dims // 2):
        a = torch.arange(first, first + n, dtype=torch.float64) * float(base) ** (-2.0 * i / dims)
        cos, sin = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        y[..., 2 * i] = u * cos - v * sin
        y[..., 2 * i + 1] = v * cos + u * sin
    return y


def attention_mixer(h, w, c, eps):
    n, H, G = h.shape[0], c["heads"], c["kv_heads"]
    q = (h @ w["q"].T + w["q.b"]).view(n, H, c["dim"])
    k = (h @ w["k"].T + w["k.b"]).view(n, G, c["dim"])
    v = (h @ w["v"].T + w["v.b"]).view(n, G, c["vdim"])
    q, k = rms_norm(q, w["q.norm"], eps), rms_norm(k, w["k.norm"], eps)
    q, k = (rotate_pairs(x, c["rot"]["dims"], c["rot"]["base"]) for x in (q, k))
    return causal_attention(q, k, v, c["scale"], w["sink"]).reshape(n, -1) @ w["o"].T


def latent_rows(h, w, eps):
    return rms_norm(h @ w["dkv"].T, w["dkv.norm"], eps)


def latent_mixer(h, w, c, latent):
    """``latent`` [n, rank]: this layer's rows or those of the layer it shares them with."""
    n, H = h.shape[0], c["heads"]
    q = (h @ w["q"].T).view(n, H, c["dim"])
    k = (latent @ w["uk"].T).view(n, H, c["dim"])
    v = (latent @ w["uv"].T).view(n, H, c["vdim"])
    o = causal_attention(q, k, v, c["scale"]).reshape(n, -1)
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


# ------------------------------------------------------------------------------------ feed-forward, head
def squared_relu(x):
    return x.clamp(min=0) ** 2


def head(x, embed, scale, cap):
    z = x @ embed.T * scale
    return cap * torch.tanh(z / cap)


# --------------------------------------------------------------------------------------- the model
def _sub(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def forward(config, weights, tokens, dtype=torch.float64, collect=None):
    """Logits [n, vocab] of one sequence; ``collect`` (a list) receives the residual after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in weights.items()}
    eps = config["norm"]["eps"]
    x = w["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    latents = {}
    for i, layer in enumerate(config["layers"]):
        lw, c = _sub(w, f"l{i}."), layer["mixer"]
        m = _sub(lw, "mix.")
        if layer["type"] == "delta":
            y = delta_mixer(x, m, c, eps)
        elif layer["type"] == "attention":
            y = attention_mixer(x, m, c, eps)
        else:
            owner = c.get("kv_from")
            if owner is None:
                latents[i] = latent_rows(x, m, eps)
            y = latent_mixer(x, m, c, latents[i if owner is None else owner])
        x = x + rms_norm(y, lw["norm1"], eps)
        if layer.get("mlp") is not None:
            x = x + rms_norm(squared_relu(x @ lw["mlp.up"].T) @ lw["mlp.down"].T, lw["norm2"], eps)
        if collect is not None:
            collect.append(x)
    return head(rms_norm(x, w["final.norm"], eps), w["embed"], config["logit_scale"], config["logit_softcap"])


def greedy(config, weights, prompt, n_new, dtype=torch.float64):
    """(generated ids, margin between the two largest logits at every generated position)."""
    ids, margins = list(prompt), []
    for _ in range(n_new):
        top = forward(config, weights, ids, dtype)[-1].topk(2)
        margins.append(float(top.values[0] - top.values[1]))
        ids.append(int(top.indices[0]))
    return ids[len(prompt):], margins
