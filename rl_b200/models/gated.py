"""Gated feed-forwards of models that are described layer by layer.

A unit is ``down(act(gate h, up h))`` with one of two activations of neighbouring columns (g, u):

    clamped to a limit     g sigmoid(1.702 g) (u + 1),  g = min(gate, limit), u = clamp(up, +-limit)
    silu (no limit)        g sigmoid(g) u

``GatedUnit`` is one unit, ``GatedExperts`` many small ones of which every token uses a few, with an optional unit for every token beside
them. Gate and up rows are interleaved in one weight (row 2i gate, row 2i + 1 up), so that a pair stands in neighbouring columns of the
product and the unit is evaluated in its epilogue. Widths are padded to multiples of 8 with zero rows and columns.

The modules' ``forward`` methods are the differentiable PyTorch statement (training, CPU); the generation engine runs the same weights
through ``rl_b200/ops/layer_ops.py``.
"""

from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn
import torch.nn.functional as TF

from .config import ModelConfig
from .mixers import _linear, pad8
from .moe import limit_groups


def clamped_glu(p: torch.Tensor, limit: float) -> torch.Tensor:
    """``p`` [..., 2 n] with gate and up in neighbouring columns -> [..., n] (fp32 inside)."""
    g, u = p[..., 0::2].float().clamp(max=limit), p[..., 1::2].float().clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)).to(p.dtype)


def silu_glu(p: torch.Tensor) -> torch.Tensor:
    return (TF.silu(p[..., 0::2].float()) * p[..., 1::2].float()).to(p.dtype)


def gated(p: torch.Tensor, limit: Optional[float]) -> torch.Tensor:
    return silu_glu(p) if limit is None else clamped_glu(p, limit)


def _limit(spec: dict) -> Optional[float]:
    return float(spec["limit"]) if spec.get("limit") is not None else None


class GatedUnit(nn.Module):
    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.ff, self.limit = spec["ff"], _limit(spec)
        d = cfg.hidden_size
        self.gate_up = nn.Parameter(torch.zeros(2 * pad8(self.ff), d, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.zeros(d, pad8(self.ff), dtype=dtype, device=device))

    def tensors(self) -> list:
        n = self.ff
        return [("gate", self.gate_up[0 : 2 * n : 2]), ("up", self.gate_up[1 : 2 * n : 2]), ("down", self.down[:, :n])]

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return _linear(gated(_linear(h, self.gate_up), self.limit), self.down)


class GatedExperts(nn.Module):
    """Sigmoid router in fp32: experts are chosen by score (+ correction) among the best groups and weighted by the scores themselves, on
    their outputs or (``weigh_input``) on their inputs, i.e. on the rows of their first product. Spec: "router", "expert", optionally
    "shared" (a unit for every token), "weigh_input", "corrected" (whether there is a correction; default yes)."""

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        r = spec["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        self.experts, self.top, self.groups, self.keep = r["experts"], r["top"], g["count"], g["keep"]
        self.ff, self.limit, self.weigh_input = spec["expert"]["ff"], _limit(spec["expert"]), bool(spec.get("weigh_input"))
        d, n = cfg.hidden_size, pad8(self.ff)
        self.router = nn.Parameter(torch.zeros(self.experts, d, dtype=dtype, device=device))
        self.gate_up = nn.Parameter(torch.zeros(self.experts, 2 * n, d, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.zeros(self.experts, d, n, dtype=dtype, device=device))
        # shifts the choice; not trained by gradient
        self.register_buffer("correction", torch.zeros(self.experts, dtype=torch.float32, device=device) if spec.get("corrected", True) else None)
        self.shared = GatedUnit(spec["shared"], cfg, dtype, device) if spec.get("shared") else None

    def tensors(self) -> list:
        n, out = self.ff, [("router", self.router)]
        if self.correction is not None:
            out.append(("correction", self.correction))
        for e in range(self.experts):
            out += [(f"e{e}.gate", self.gate_up[e, 0 : 2 * n : 2]), (f"e{e}.up", self.gate_up[e, 1 : 2 * n : 2]), (f"e{e}.down", self.down[e, :, :n])]
        return out + ([(f"shared.{leaf}", t) for leaf, t in self.shared.tensors()] if self.shared is not None else [])

    def choose(self, z: torch.Tensor):
        """Router logits [T, experts] fp32 -> (weights, expert ids) [T, top]."""
        s = torch.sigmoid(z)
        c = s if self.correction is None else s + self.correction
        idx = limit_groups(c, self.groups, self.keep, float("-inf")).topk(self.top, dim=-1)[1]
        return s.gather(1, idx), idx

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        w, idx = self.choose(h.float() @ self.router.float().t())
        y = torch.zeros(h.shape, dtype=torch.float32, device=h.device) if self.shared is None else self.shared(h).float()
        for e in range(self.experts):
            tok, slot = (idx == e).nonzero(as_tuple=True)
            if tok.numel():
                p, wt = TF.linear(h[tok], self.gate_up[e]), w[tok, slot, None]
                a = gated((p.float() * wt).to(p.dtype) if self.weigh_input else p, self.limit)
                o = TF.linear(a, self.down[e]).float()
                y = y.index_add(0, tok, o if self.weigh_input else o * wt)
        return y


def feed_forward(spec: dict, cfg: ModelConfig, dtype, device) -> nn.Module:
    return (GatedExperts if spec["kind"] == "moe" else GatedUnit)(spec, cfg, dtype, device)
