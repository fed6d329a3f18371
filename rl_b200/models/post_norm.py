"""The layer whose sublayers run one after the other on the residual stream itself, their outputs normed before they join it:

    x <- x + m norm1(mixer(x));   x <- x + m norm2(feed-forward(x));   x <- x + m norm(proj(gelu(gate x) * e[token]))

The last line is the layer's token input: a table row per token and layer (``CausalLM.side_embed`` holds all layers' columns side by
side), gated by the stream. The feed-forward (or the token input) may be absent. The residual stream and the norms are fp32, ``m`` is
the configuration's residual multiplier.

Feed-forwards are gated units with clamped inputs, ``g sigmoid(1.702 g) (u + 1)`` with g = min(gate, limit), u = clamp(up, +-limit): one
(``ClampedGLU``) or many small ones of which every token uses a few (``ClampedExperts``). Gate and up rows are interleaved in one weight
(row 2i gate, row 2i + 1 up), so that a pair stands in neighbouring columns of the product and the unit is evaluated in its epilogue.
Widths are padded to multiples of 8 with zero rows and columns.

The modules' ``forward`` methods are the differentiable PyTorch statement (training, CPU); the generation engine runs the same weights
through ``rl_b200/ops/layer_ops.py``.
"""

from __future__ import annotations

import torch
import torch.nn as nn
import torch.nn.functional as TF

from .config import ModelConfig
from .mixers import MIXERS, _linear, pad8, rms_unit
from .moe import limit_groups


def clamped_glu(p: torch.Tensor, limit: float) -> torch.Tensor:
    """``p`` [..., 2 n] with gate and up in neighbouring columns -> [..., n] (fp32 inside)."""
    g, u = p[..., 0::2].float().clamp(max=limit), p[..., 1::2].float().clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)).to(p.dtype)


class ClampedGLU(nn.Module):
    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.ff, self.limit = spec["ff"], float(spec["limit"])
        d = cfg.hidden_size
        self.gate_up = nn.Parameter(torch.zeros(2 * pad8(self.ff), d, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.zeros(d, pad8(self.ff), dtype=dtype, device=device))

    def tensors(self) -> list:
        n = self.ff
        return [("gate", self.gate_up[0 : 2 * n : 2]), ("up", self.gate_up[1 : 2 * n : 2]), ("down", self.down[:, :n])]

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return _linear(clamped_glu(_linear(h, self.gate_up), self.limit), self.down)


class ClampedExperts(nn.Module):
    """Sigmoid router in fp32: experts are chosen by score + correction among the best groups, weighted by the scores themselves."""

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        r = spec["router"]
        g = r.get("groups") or {"count": 1, "keep": 1}
        self.experts, self.top, self.groups, self.keep = r["experts"], r["top"], g["count"], g["keep"]
        self.ff, self.limit = spec["expert"]["ff"], float(spec["expert"]["limit"])
        d, n = cfg.hidden_size, pad8(self.ff)
        self.router = nn.Parameter(torch.zeros(self.experts, d, dtype=dtype, device=device))
        self.gate_up = nn.Parameter(torch.zeros(self.experts, 2 * n, d, dtype=dtype, device=device))
        self.down = nn.Parameter(torch.zeros(self.experts, d, n, dtype=dtype, device=device))
        self.register_buffer("correction", torch.zeros(self.experts, dtype=torch.float32, device=device))   # shifts the choice; not trained by gradient

    def tensors(self) -> list:
        n, out = self.ff, [("router", self.router), ("correction", self.correction)]
        for e in range(self.experts):
            out += [(f"e{e}.gate", self.gate_up[e, 0 : 2 * n : 2]), (f"e{e}.up", self.gate_up[e, 1 : 2 * n : 2]), (f"e{e}.down", self.down[e, :, :n])]
        return out

    def choose(self, z: torch.Tensor):
        """Router logits [T, experts] fp32 -> (weights, expert ids) [T, top]."""
        s = torch.sigmoid(z)
        idx = limit_groups(s + self.correction, self.groups, self.keep, float("-inf")).topk(self.top, dim=-1)[1]
        return s.gather(1, idx), idx

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        w, idx = self.choose(h.float() @ self.router.float().t())
        y = torch.zeros(h.shape, dtype=torch.float32, device=h.device)
        for e in range(self.experts):
            tok, slot = (idx == e).nonzero(as_tuple=True)
            if tok.numel():
                o = TF.linear(clamped_glu(TF.linear(h[tok], self.gate_up[e]), self.limit), self.down[e])
                y = y.index_add(0, tok, o.float() * w[tok, slot, None])
        return y


class PostNormBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype, device, tp=None, ep=None, cp=None, lora=None, layer_idx: int = 0):
        super().__init__()
        assert (tp is None or tp.world == 1) and (cp is None or cp.world == 1) and not lora, "post-norm layers: no tensor / context parallelism, no LoRA"
        self.cfg, self.layer_idx, self.window = cfg, layer_idx, 0
        entry, d = cfg.mixers[layer_idx], cfg.hidden_size
        norm = lambda: nn.Parameter(torch.ones(d, dtype=dtype, device=device))   # noqa: E731
        self.mixer = MIXERS[entry["type"]](entry["mixer"], cfg, dtype, device)
        self.norm1 = norm()
        self.ff = None
        if entry.get("mlp"):
            self.ff = (ClampedExperts if entry["mlp"]["kind"] == "moe" else ClampedGLU)(entry["mlp"], cfg, dtype, device)
            self.norm2 = norm()
        self.side_dim = cfg.token_side["dim"] if cfg.token_side else 0
        if self.side_dim:
            self.side_gate = nn.Parameter(torch.zeros(pad8(self.side_dim), d, dtype=dtype, device=device))
            self.side_proj = nn.Parameter(torch.zeros(d, pad8(self.side_dim), dtype=dtype, device=device))
            self.side_norm = norm()
        self.self_attn = self.mlp = None                   # (the names other families' walkers look for)

    def tensor_views(self, prefix: str) -> list:
        """(checkpoint name, view of a parameter) of every tensor of this layer."""
        out = [(f"{prefix}norm1", self.norm1)] + [(f"{prefix}mix.{leaf}", t) for leaf, t in self.mixer.tensors()]
        if self.ff is not None:
            out += [(f"{prefix}norm2", self.norm2)] + [(f"{prefix}mlp.{leaf}", t) for leaf, t in self.ff.tensors()]
        if self.side_dim:
            n = self.side_dim
            out += [(f"{prefix}side.gate", self.side_gate[:n]), (f"{prefix}side.proj", self.side_proj[:, :n]), (f"{prefix}side.norm", self.side_norm)]
        return out

    def join(self, x: torch.Tensor, y: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        c = self.cfg
        return x + c.residual_mult * (rms_unit(y.float(), c.rms_norm_eps) * w.float())

    def forward(self, x, positions, side, cu_seqlens, max_seqlen):
        """``side`` [T, side_dim]: the tokens' rows of this layer's part of the table (None: no token input)."""
        dt, m = self.norm1.dtype, self.mixer
        bias = lambda y, b: y if b is None else y + b   # noqa: E731
        y = m.sequence(bias(_linear(x.to(dt), m.in_proj), m.in_bias), positions, cu_seqlens)
        y = TF.pad(y, (0, m.mix_width - y.shape[1]))
        x = self.join(x, bias(_linear(y, m.out_proj), m.out_bias), self.norm1)
        if self.ff is not None:
            x = self.join(x, self.ff(x.to(dt)), self.norm2)
        if self.side_dim:
            g = TF.gelu(_linear(x.to(dt), self.side_gate).float(), approximate="tanh")[:, : self.side_dim] * side.float()
            x = self.join(x, _linear(TF.pad(g, (0, self.side_gate.shape[0] - self.side_dim)).to(dt), self.side_proj), self.side_norm)
        return x
