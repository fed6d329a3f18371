"""Plain, slow statement of the Gadarax decoder in float64: one function per mechanism, one sequence at a time, no cache and no
batching. The tests compare the framework with it; it shares no code with the framework.

A model is a configuration dictionary in the ``config.json`` layout and a dictionary of tensors under their checkpoint names.
"""

from __future__ import annotations

import math

import torch

D = torch.float64


def dyt(x, w, b, alpha):
    """Dynamic tanh: y = w * tanh(alpha x) + b."""
    return torch.tanh(alpha * x) * w + b


def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def frequencies(rot):
    """(angle per position of every pair, factor on cos and sin)."""
    n, base = rot["dims"], rot["base"]
    f = [base ** (-2.0 * i / n) for i in range(n // 2)]
    s = rot.get("scaling")
    if not s:
        return f, 1.0

    def turn_dim(t):
        return n * math.log(s["original"] / (2 * math.pi * t)) / (2 * math.log(base))

    lo = max(math.floor(turn_dim(s["fast"])), 0)
    hi = min(math.ceil(turn_dim(s["slow"])), n - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / s["factor"] * r + fi * (1 - r))
    return out, 0.1 * math.log(s["factor"]) + 1.0


def rotate(x, rot, first, interleaved):
    """x [T, H, n]: rotates the leading rot.dims entries of every head; row t stands at position first + t."""
    f, m = frequencies(rot)
    y = x.clone()
    n = rot["dims"]
    for i, fi in enumerate(f):
        a, b = (2 * i, 2 * i + 1) if interleaved else (i, i + n // 2)
        ang = torch.arange(first, first + x.shape[0], dtype=D)[:, None] * fi
        c, s = torch.cos(ang) * m, torch.sin(ang) * m
        y[:, :, a] = x[:, :, a] * c - x[:, :, b] * s
        y[:, :, b] = x[:, :, b] * c + x[:, :, a] * s
    return y


def latent_attention(w, h, m, eps):
    """w: name -> tensor below '<layer>.mix.'."""
    T, H, dn, dr, dv, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = (h @ w["q"].T).view(T, H, dn + dr)
    lat = h @ w["dkv"].T
    c = unit_rms(lat[:, :R], eps) * w["dkv.norm"]
    k_rot = rotate(lat[:, R:].view(T, 1, dr), m["rot"], 0, True)
    q_rot = rotate(q[:, :, dn:], m["rot"], 0, True)
    k = (c @ w["uk"].T).view(T, H, dn)
    v = (c @ w["uv"].T).view(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for i in range(T):
        for hd in range(H):
            s = (k[: i + 1, hd] @ q[i, hd, :dn] + k_rot[: i + 1, 0] @ q_rot[i, hd]) * m["scale"]
            p = torch.softmax(s, 0)
            out[i, hd] = p @ v[: i + 1, hd]
    gate = torch.sigmoid(h @ w["g"].T)
    return (out.reshape(T, H * dv) * gate) @ w["o"].T


def retention(w, h, m, eps, state=None):
    """Token by token. Returns the mixer's output and the state [heads, dim, vdim] after the last token."""
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rotate((h @ w["q"].T).view(T, H, dk), m["rot"], 0, False)
    k = rotate((h @ w["k"].T).view(T, H, dk), m["rot"], 0, False) * dk ** -0.5
    v = (h @ w["v"].T).view(T, H, dv)
    decay = torch.tensor(m["decay"], dtype=h.dtype)
    S = torch.zeros(H, dk, dv, dtype=h.dtype) if state is None else state
    out = torch.zeros(T, H, dv, dtype=h.dtype)
    for t in range(T):
        S = decay[:, None, None] * S + k[t, :, :, None] * v[t, :, None, :]
        out[t] = (S * q[t, :, :, None]).sum(1)
    y = unit_rms(out, eps).reshape(T, H * dv)
    g = h @ w["g"].T
    return (y * (g * torch.sigmoid(g))) @ w["o"].T, S


def feed_forward(w, h):
    u = torch.relu(h @ w["up"].T)
    return (u * u) @ w["down"].T


def run_order(cfg):
    """(layer, pass or None) in the order the layers run."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if not lp:
        return [(i, None) for i in range(n)]
    out = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        out += [(i, t) for i in range(lp["start"], lp["stop"])]
    return out + [(i, None) for i in range(lp["stop"], n)]


def below(weights, prefix):
    return {k[len(prefix) :]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence; ``layers_out``: a list that receives the residual after every layer run."""
    W = {k: v.to(D) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    e = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] * cfg["embedding"]["scale"]
    x = e.clone()
    for i, t in run_order(cfg):
        if t is not None and i == cfg["loop"]["start"]:
            if t > 0:
                x = x + e
            x = x + W["loop.step"][t]
        spec = cfg["layers"][i]
        h = dyt(x, W[f"l{i}.norm1"], W[f"l{i}.norm1.b"], W[f"l{i}.norm1.alpha"])
        mix = below(W, f"l{i}.mix.")
        if spec["type"] == "latent_attention":
            y = latent_attention(mix, h, spec["mixer"], eps)
        else:
            y, _ = retention(mix, h, spec["mixer"], eps)
        if spec.get("mlp"):
            y = y + feed_forward(below(W, f"l{i}.mlp."), h)
        x = x + y
        if layers_out is not None:
            layers_out.append(x.clone())
    return dyt(x, W["final.norm"], W["final.norm.b"], W["final.norm.alpha"]) @ W["embed"].T
