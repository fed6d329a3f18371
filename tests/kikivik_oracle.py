"""Plain, slow statement of the Kikivik decoder in float64: one function per mechanism, one sequence at a time, no cache and no batching.
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


def frequencies(rot):
    """Angle per position of every pair; slowed down by the scaling factor where there is one."""
    n = rot["dims"]
    f = [rot["base"] ** (-2.0 * i / n) for i in range(n // 2)]
    return [x / rot["scaling"]["factor"] for x in f] if rot.get("scaling") else f


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


def visible(T, size=None):
    """[T, T]: whether row i sees column j: not behind itself and, in chunks of ``size`` from position 0, in its own chunk."""
    i = torch.arange(T)
    seen = i[None, :] <= i[:, None]
    return seen if size is None else seen & (i[None, :] // size == i[:, None] // size)


def attend(q, k, v, scale, seen):
    """One head: q, k [T, dim], v [T, vdim]."""
    s = (q @ k.T * scale).masked_fill(~seen, -math.inf)
    return torch.softmax(s, -1) @ v


def latent_attention(w, h, m, eps):
    T, H, dk, dr, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    cq = rms(h @ w["dq"].T, eps) * w["dq.norm"]
    q = (cq @ w["uq"].T).view(T, H, dk + dr)
    low = h @ w["dkv"].T
    c = rms(low[:, : m["kv_rank"]], eps) * w["dkv.norm"]
    kr = rotate(low[:, None, m["kv_rank"] :], m["rot"])[:, 0]
    k, v = (c @ w["uk"].T).view(T, H, dk), (c @ w["uv"].T).view(T, H, dv)
    q = torch.cat([q[:, :, :dk], rotate(q[:, :, dk:], m["rot"])], -1)
    out = torch.stack([attend(q[:, i], torch.cat([k[:, i], kr], -1), v[:, i], m["scale"], visible(T)) for i in range(H)], 1)
    return out.reshape(T, H * dv) @ w["o"].T


def mix_values(v, first, share):
    """Part ``share`` of the first layer's values replaces as much of the layer's own."""
    return (1 - share) * v + share * first


def attention(w, h, m, eps, values):
    """``values``: a list that holds the values of the first layer that mixes them, once there was one."""
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate(rms((h @ w["q"].T).view(T, H, dk), eps) * w["q.norm"], m["rot"])
    k = rotate(rms((h @ w["k"].T).view(T, G, dk), eps) * w["k.norm"], m["rot"])
    v = (h @ w["v"].T).view(T, G, dv)
    if m.get("v_mix"):
        if values:
            v = mix_values(v, values[0], w["vmix"])
        else:
            values.append(v)
    size = m["mask"]["size"] if m.get("mask") else None
    out = torch.stack([attend(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], m["scale"], visible(T, size)) for i in range(H)], 1)
    return out.reshape(T, H * dv) @ w["o"].T


def clamped_unit(w, h, limit):
    g, u = torch.clamp(h @ w["gate"].T, max=limit), torch.clamp(h @ w["up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ w["down"].T


def silu_unit(w, h):
    g = h @ w["gate"].T
    return (g * sigmoid(g) * (h @ w["up"].T)) @ w["down"].T


def route(w, h, r):
    """Chosen experts and their weights, per token: lists of (expert, weight)."""
    s = sigmoid(h @ w["router"].T)
    return [[(e, s[t, e]) for e in sorted(range(r["experts"]), key=lambda e: -float(s[t, e]))[: r["top"]]] for t in range(h.shape[0])]


def experts(w, h, mlp):
    """An expert reads its token's row times the router's weight."""
    y = torch.zeros_like(h)
    for t, chosen in enumerate(route(w, h, mlp["router"])):
        for e, weight in chosen:
            y[t] += silu_unit(below(w, f"e{e}."), weight * h[t : t + 1])[0]
    return y + silu_unit(below(w, "shared."), h) if mlp.get("shared") else y


def feed_forward(w, h, mlp):
    return experts(w, h, mlp) if mlp["kind"] == "moe" else clamped_unit(w, h, mlp["limit"])


def below(weights, prefix):
    return {k[len(prefix) :]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual stream after every layer."""
    W = {k: v.to(D) for k, v in weights.items()}
    eps, values = cfg["norm"]["eps"], []
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    for i, spec in enumerate(cfg["layers"]):
        w, h = below(W, f"l{i}.mix."), rms(x, eps) * W[f"l{i}.norm1"]
        x = x + (attention(w, h, spec["mixer"], eps, values) if spec["type"] == "attention" else latent_attention(w, h, spec["mixer"], eps))
        if spec.get("mlp"):
            x = x + feed_forward(below(W, f"l{i}.mlp."), rms(x, eps) * W[f"l{i}.norm2"], spec["mlp"])
        if layers_out is not None:
            layers_out.append(x.clone())
    return rms(x, eps) * W["final.norm"] @ W["head"].T
