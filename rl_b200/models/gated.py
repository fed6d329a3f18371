"""Feed-forwards of models that are described layer by layer.

A gated unit is ``down(act(gate h, up h))`` with one of two activations of neighbouring columns (g, u):

    clamped to a limit     g sigmoid(1.702 g) (u + 1),  g = min(gate, limit), u = clamp(up, +-limit)
    silu (no limit)        g sigmoid(g) u

``GatedUnit`` is one unit, ``GatedExperts`` many small ones of which every token uses a few, with an optional unit for every token beside
them. ``PolyUnit`` is ``down(act(up h))`` with a polynomial of normed powers as its activation. Gate and up rows are interleaved in one weight (row 2i gate, row 2i + 1 up), so that a pair stands in neighbouring columns of the
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
from .mixers import _linear, pad8, rms_unit
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


def poly_norm(z: torch.Tensor, coef: torch.Tensor, eps: float) -> torch.Tensor:
    """c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3 with N(y) = y over the root mean square of its row, in fp32. For every row that is one cubic
    polynomial of the entries."""
    z, c = z.float(), coef.float()
    y = c[3]
    for i in range(3):
        y = y + c[i] * rms_unit(z ** (i + 1), eps)
    return y


class PolyUnit(nn.Module):
    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.ff, self.eps = spec["ff"], cfg.rms_norm_eps
        d, n = cfg.hidden_size, pad8(self.ff)
        self.up = nn.Parameter(torch.zeros(n, d, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.zeros(d, n, dtype=dtype, device=device))
        self.coef = nn.Parameter(torch.tensor([1 / 3, 1 / 3, 1 / 3, 0.0], dtype=dtype, device=device))

    def tensors(self) -> list:
        return [("up", self.up[: self.ff]), ("down", self.down[:, : self.ff]), ("act", self.coef)]

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        p = _linear(h, self.up)
        a = poly_norm(p[:, : self.ff], self.coef, self.eps).to(p.dtype)
        return _linear(TF.pad(a, (0, p.shape[1] - self.ff)), self.down)


class GatedExperts(nn.Module):
    """Router in fp32: experts are chosen by score (+ correction) among the best groups and weighted by the scores themselves (times a
    constant), on their outputs or (``weigh_input``) on their inputs, i.e. on the rows of their first product. Spec: "router" ("experts", "top",
    optionally "groups", "scale", "identity": that many more outputs, behind the experts', which stand for the input itself), "expert",
    optionally "shared" (a unit for every token), "shared_gate" (its output is multiplied by a sigmoid, one number per token), "score" ("sigmoid",
    the default, or "softmax" over all outputs), "weigh_input", "corrected" (whether there is a correction; default yes)."""

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        r = spec["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        self.experts, self.top, self.groups, self.keep = r["experts"], r["top"], g["count"], g["keep"]
        self.ff, self.limit, self.weigh_input = spec["expert"]["ff"], _limit(spec["expert"]), bool(spec.get("weigh_input"))
        d, n = cfg.hidden_size, pad8(self.ff)
        self.identity, self.scale, self.softmax = r.get("identity", 0), float(r.get("scale", 1.0)), spec.get("score", "sigmoid") == "softmax"
        self.outputs = self.experts + self.identity
        self.shared_gate = bool(spec.get("shared") and spec.get("shared_gate"))
        assert not (self.weigh_input and self.identity), "weights on the experts' inputs and identity outputs"
        # the shared unit's gate is one more row behind the outputs
        rows = self.outputs + int(self.shared_gate)
        self.router = nn.Parameter(torch.zeros(rows if rows == self.experts else pad8(rows), d, dtype=dtype, device=device))
        self.gate_up = nn.Parameter(torch.zeros(self.experts, 2 * n, d, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.zeros(self.experts, d, n, dtype=dtype, device=device))
        # shifts the choice; not trained by gradient
        self.register_buffer("correction", torch.zeros(self.outputs, dtype=torch.float32, device=device) if spec.get("corrected", True) else None)
        self.shared = GatedUnit(spec["shared"], cfg, dtype, device) if spec.get("shared") else None

    def tensors(self) -> list:
        n, out = self.ff, [("router", self.router[: self.outputs])]
        if self.correction is not None:
            out.append(("correction", self.correction))
        for e in range(self.experts):
            out += [(f"e{e}.gate", self.gate_up[e, 0 : 2 * n : 2]), (f"e{e}.up", self.gate_up[e, 1 : 2 * n : 2]), (f"e{e}.down", self.down[e, :, :n])]
        if self.shared_gate:
            out.append(("shared.sg", self.router[self.outputs : self.outputs + 1]))
        return out + ([(f"shared.{leaf}", t) for leaf, t in self.shared.tensors()] if self.shared is not None else [])

    def choose(self, z: torch.Tensor):
        """Router logits [T, outputs] fp32 -> (weights, indices) [T, top]."""
        s = torch.softmax(z, -1) if self.softmax else torch.sigmoid(z)
        c = s if self.correction is None else s + self.correction
        idx = limit_groups(c, self.groups, self.keep, float("-inf")).topk(self.top, dim=-1)[1]
        return s.gather(1, idx) * self.scale, idx

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        z = h.float() @ self.router.float().t()
        w, idx = self.choose(z[:, : self.outputs])
        y = torch.zeros(h.shape, dtype=torch.float32, device=h.device) if self.shared is None else self.shared(h).float()
        if self.shared_gate:
            y = y * torch.sigmoid(z[:, self.outputs, None])
        if self.identity:
            y = y + h.float() * (w * (idx >= self.experts)).sum(-1, keepdim=True)
        for e in range(self.experts):
            tok, slot = (idx == e).nonzero(as_tuple=True)
            if tok.numel():
                p, wt = TF.linear(h[tok], self.gate_up[e]), w[tok, slot, None]
                a = gated((p.float() * wt).to(p.dtype) if self.weigh_input else p, self.limit)
                o = TF.linear(a, self.down[e]).float()
                y = y.index_add(0, tok, o if self.weigh_input else o * wt)
        return y


def feed_forward(spec: dict, cfg: ModelConfig, dtype, device) -> nn.Module:
    kind = GatedExperts if spec["kind"] == "moe" else PolyUnit if spec.get("act") == "poly" else GatedUnit
    return kind(spec, cfg, dtype, device)
