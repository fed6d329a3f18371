"""Plain, slow statement of the Zonidra decoder in float64: one function per mechanism, one sequence at a time, no cache and no batching.
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


def sigmoid(x):
    return 1 / (1 + torch.exp(-x))


def pair_rows(tokens, bigram):
    """Row of the pair table for every token: a hash of the token before and the token; the last row for the first token."""
    return [bigram["buckets"] if i == 0 else (tokens[i - 1] * bigram["mul_prev"] + t * bigram["mul_cur"]) % bigram["buckets"] for i, t in enumerate(tokens)]


def shift(h, s):
    """Every row moves by the share s (per element) towards the row before it; the first one towards zero."""
    before = torch.cat([torch.zeros_like(h[:1]), h[:-1]])
    return h + (before - h) * s


def frequencies(rot):
    """Angle per position of every pair. Scaled: turns with a wavelength above original / low are slowed down by the factor, those below
    original / high stay, between them the two mix linearly in original / wavelength."""
    n, s = rot["dims"], rot.get("scaling")
    out = []
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        if s:
            length = 2 * math.pi / f
            if length > s["original"] / s["low"]:
                f = f / s["factor"]
            elif length >= s["original"] / s["high"]:
                t = (s["original"] / length - s["low"]) / (s["high"] - s["low"])
                f = (1 - t) * f / s["factor"] + t * f
        out.append(f)
    return out


def rotate(x, rot, first=0):
    """x [T, H, n]; of the leading rot.dims entries, entry i and entry i + dims / 2 turn by position * frequency i."""
    half = rot["dims"] // 2
    y = x.clone()
    for i, f in enumerate(frequencies(rot)):
        a = torch.arange(first, first + x.shape[0], dtype=x.dtype)[:, None] * f
        u, v = x[:, :, i], x[:, :, i + half]
        y[:, :, i] = u * torch.cos(a) - v * torch.sin(a)
        y[:, :, i + half] = v * torch.cos(a) + u * torch.sin(a)
    return y


def visible(T, mask=None):
    """[T, T]: whether row i sees column j: not behind itself, and nearer than the window's size or among the first tokens that are kept."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    seen = j <= i
    return seen & ((i - j < mask["size"]) | (j < mask.get("keep_first", 0))) if mask else seen


def attend(q, k, v, scale, offset, seen):
    """One head: q, k [T, dim], v [T, vdim]. Every visible key weighs sigmoid(score + offset), whatever the others weigh."""
    return torch.where(seen, sigmoid(q @ k.T * scale + offset), torch.zeros((), dtype=q.dtype)) @ v


def keys_values(w, h, m):
    T, G = h.shape[0], m["kv_heads"]
    return rotate((h @ w["k"].T).view(T, G, m["dim"]), m["rot"]), (h @ w["v"].T).view(T, G, m["vdim"])


def attention(w, h, m, kv=None):
    """``kv``: another layer's keys and values (None: the layer's own). Returns (output, keys and values)."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    k, v = kv if kv is not None else keys_values(w, h, m)
    q = rotate((h @ w["q"].T).view(T, H, m["dim"]), m["rot"])
    seen = visible(T, m.get("mask"))
    out = torch.stack([attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], w["pb"][i], seen) for i in range(H)], 1)
    return (out.reshape(T, H * m["vdim"]) * sigmoid(h @ w["g"].T)) @ w["o"].T, (k, v)


def poly_norm(z, coef, eps):
    a, b, c, e = coef
    return a * rms(z, eps) + b * rms(z * z, eps) + c * rms(z * z * z, eps) + e


def poly_unit(w, h, eps):
    return poly_norm(h @ w["up"].T, w["act"], eps) @ w["down"].T


def silu_unit(w, h):
    g = h @ w["gate"].T
    return (g * sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def route(w, h, r):
    """Chosen outputs of the router and their weights, per token: lists of (index, weight)."""
    s = torch.softmax(h @ w["router"].T, -1)
    c = s + w["correction"]
    n = r["experts"] + r.get("identity", 0)
    return [[(e, s[t, e] * r.get("scale", 1.0)) for e in sorted(range(n), key=lambda e: -float(c[t, e]))[: r["top"]]] for t in range(h.shape[0])]


def experts(w, h, mlp):
    """Router outputs behind the experts stand for the token's own row."""
    y = torch.zeros_like(h)
    for t, chosen in enumerate(route(w, h, mlp["router"])):
        for e, weight in chosen:
            y[t] += weight * (h[t] if e >= mlp["router"]["experts"] else silu_unit(below(w, f"e{e}."), h[t : t + 1])[0])
    if mlp.get("shared"):
        y = y + sigmoid(h @ w["shared.sg"].T) * silu_unit(below(w, "shared."), h)
    return y


def feed_forward(w, h, mlp, eps):
    return experts(w, h, mlp) if mlp["kind"] == "moe" else poly_unit(w, h, eps)


def below(weights, prefix):
    return {k[len(prefix) :]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer."""
    W = {k: v.to(D) for k, v in weights.items()}
    eps, kv = cfg["norm"]["eps"], {}
    tokens = [int(t) for t in tokens]
    x = W["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    if cfg["embedding"].get("bigram"):
        x = x + W["bigram"][torch.tensor(pair_rows(tokens, cfg["embedding"]["bigram"]))]
    for i, spec in enumerate(cfg["layers"]):
        L, m = below(W, f"l{i}."), spec["mixer"]
        h = shift(rms(x, eps) * L["norm1"], L["shift"])
        y, kv[i] = attention(below(L, "mix."), h, m, kv[m["kv_from"]] if m.get("kv_from") is not None else None)
        x = x + rms(y, eps) * L["norm1b"] * L["ls1"]
        if spec.get("mlp"):
            y = feed_forward(below(L, "mlp."), rms(x, eps) * L["norm2"], spec["mlp"], eps)
            x = x + rms(y, eps) * L["norm2b"] * L["ls2"]
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps) * W["final.norm"] @ W["head"].T
