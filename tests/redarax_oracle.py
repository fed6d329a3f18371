"""Plain, slow statement of the Redarax decoder in float64: one function per mechanism, one sequence at a time, no cache and no batching.
The tests compare the framework with it; it shares no code with the framework.

A model is a configuration dictionary in the ``config.json`` layout and a dictionary of tensors under their checkpoint names. ``w`` below
is the dictionary of one module's tensors without the module's prefix.
"""

from __future__ import annotations

import math

import torch

D = torch.float64


def rms(x, eps):
    """x over its root mean square, along the last dimension."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(x):
    return x / (1 + torch.exp(-x))


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def softplus(x):
    return torch.logaddexp(x, torch.zeros_like(x))


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def rotate(x, rot, first=0):
    """x [T, H, n]; pair (2i, 2i + 1) of the leading rot.dims entries turns by position * base^(-2i / dims)."""
    n = rot["dims"]
    y = x.clone()
    for i in range(n // 2):
        a = torch.arange(first, first + x.shape[0], dtype=x.dtype)[:, None] * rot["base"] ** (-2.0 * i / n)
        u, v = x[:, :, 2 * i], x[:, :, 2 * i + 1]
        y[:, :, 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        y[:, :, 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return y


def attention(w, h, m, eps):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T + w["q.b"]).view(T, H, dk)
    k = (h @ w["k"].T + w["k.b"]).view(T, G, dk)
    v = (h @ w["v"].T + w["v.b"]).view(T, G, dv)
    q = rotate(rms(q, eps) * w["q.norm"], m["rot"])
    k = rotate(rms(k, eps) * w["k.norm"], m["rot"])
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        s = q[:, hd] @ k[:, g].T * m["scale"]
        s = s.masked_fill(torch.ones(T, T, dtype=torch.bool).triu(1), -math.inf)
        out[:, hd] = torch.softmax(s, -1) @ v[:, g]
    return out.reshape(T, H * dv) @ w["o"].T + w["o.b"]


def short_conv(x, taps, bias=None):
    """x [T, C], taps [C, n]: y_t = sum_j taps[:, j] x_(t - n + 1 + j), zeros before the start."""
    T, n = x.shape[0], taps.shape[1]
    y = torch.zeros_like(x)
    for t in range(T):
        for j in range(n):
            s = t - n + 1 + j
            if s >= 0:
                y[t] += taps[:, j] * x[s]
    return y if bias is None else y + bias


def mamba2(w, h, m, eps):
    T, H, P, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], -1)
    xbc = silu(short_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = xbc[:, :inner].view(T, H, P), xbc[:, inner : inner + G * N].view(T, G, N), xbc[:, inner + G * N :].view(T, G, N)
    dt = softplus(dt + w["dt_bias"])
    A = -torch.exp(w["A_log"])
    S = torch.zeros(H, N, P, dtype=h.dtype)
    y = torch.zeros(T, H, P, dtype=h.dtype)
    for t in range(T):
        for hd in range(H):
            g = hd // (H // G)
            S[hd] = torch.exp(A[hd] * dt[t, hd]) * S[hd] + dt[t, hd] * torch.outer(B[t, g], x[t, hd])
            y[t, hd] = S[hd].T @ C[t, g] + w["D"][hd] * x[t, hd]
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * w["norm"]
    return y @ w["o"].T


def delta(w, h, m, eps):
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = silu(short_conv(h @ w["q"].T, w["q.conv"])).view(T, G, dk)
    k = silu(short_conv(h @ w["k"].T, w["k.conv"])).view(T, G, dk)
    v = silu(short_conv(h @ w["v"].T, w["v.conv"])).view(T, H, dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * dk ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    beta = sigmoid(h @ w["b"].T)
    decay = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for hd in range(H):
        g = hd // (H // G)
        S = torch.zeros(dk, dv, dtype=h.dtype)
        for t in range(T):
            S = decay[t, hd] * S
            u = beta[t, hd] * (v[t, hd] - S.T @ k[t, g])
            S = S + torch.outer(k[t, g], u)
            out[t, hd] = S.T @ q[t, g]
    y = rms(out, eps) * w["norm"] * silu((h @ w["g"].T).view(T, H, dv))
    return y.reshape(T, H * dv) @ w["o"].T


MIXERS = {"attention": attention, "mamba2": mamba2, "delta": delta}


def clamped_glu(w, h, limit):
    g = torch.clamp(h @ w["gate"].T, max=limit)
    u = torch.clamp(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


def route(w, h, r):
    """Chosen experts and their weights, per token: lists of (expert, weight)."""
    s = sigmoid(h @ w["router"].T)
    choice = s + w["correction"]
    E, groups = r["experts"], r.get("groups") or {"count": 1, "keep": 1}
    size = E // groups["count"]
    out = []
    for t in range(h.shape[0]):
        c = choice[t].tolist()
        rank = sorted(range(groups["count"]), key=lambda g: -sum(sorted(c[g * size : (g + 1) * size])[-2:]))
        keep = set(rank[: groups["keep"]])
        order = sorted((e for e in range(E) if e // size in keep), key=lambda e: -c[e])
        out.append([(e, s[t, e]) for e in order[: r["top"]]])
    return out


def experts(w, h, mlp):
    y = torch.zeros_like(h)
    for t, chosen in enumerate(route(w, h, mlp["router"])):
        for e, weight in chosen:
            y[t] += weight * clamped_glu(below(w, f"e{e}."), h[t : t + 1], mlp["expert"]["limit"])[0]
    return y


def feed_forward(w, h, mlp):
    return experts(w, h, mlp) if mlp["kind"] == "moe" else clamped_glu(w, h, mlp["limit"])


def token_side(w, x, e, eps):
    y = (gelu_tanh(x @ w["gate"].T) * e) @ w["proj"].T
    return rms(y, eps) * w["norm"]


def below(weights, prefix):
    return {k[len(prefix) :]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer."""
    W = {k: v.to(D) for k, v in weights.items()}
    eps, m = cfg["norm"]["eps"], cfg["residual_mult"]
    ids = torch.as_tensor(tokens, dtype=torch.long)
    x = W["embed"][ids]
    for i, spec in enumerate(cfg["layers"]):
        x = x + m * rms(MIXERS[spec["type"]](below(W, f"l{i}.mix."), x, spec["mixer"], eps), eps) * W[f"l{i}.norm1"]
        if spec.get("mlp"):
            x = x + m * rms(feed_forward(below(W, f"l{i}.mlp."), x, spec["mlp"]), eps) * W[f"l{i}.norm2"]
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = x + m * token_side(below(W, f"l{i}.side."), x, W["side.embed"][ids, i * n : (i + 1) * n], eps)
        if layers_out is not None:
            layers_out.append(x.clone())
    z = rms(x, eps) * W["final.norm"] @ W["head"].T * cfg["logit_scale"]
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
