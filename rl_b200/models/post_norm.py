"""The layer whose sublayers run one after the other on the residual stream itself, their outputs normed before they join it:

    x <- x + m norm1(mixer(x));   x <- x + m norm2(feed-forward(x));   x <- x + m norm(proj(gelu(gate x) * e[token]))

The last line is the layer's token input: a table row per token and layer (``CausalLM.side_embed`` holds all layers' columns side by
side), gated by the stream. The feed-forward (or the token input) may be absent. The residual stream and the norms are fp32, ``m`` is
the configuration's residual multiplier.

Feed-forwards are gated units with clamped inputs, or experts of such units (``gated.py``).

The modules' ``forward`` methods are the differentiable PyTorch statement (training, CPU); the generation engine runs the same weights
through ``rl_b200/ops/layer_ops.py``.
"""

from __future__ import annotations

import torch
import torch.nn as nn
import torch.nn.functional as TF

from .config import ModelConfig
from .gated import feed_forward
from .mixers import MIXERS, _linear, pad8, rms_unit


class PostNormBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype, device, tp=None, ep=None, cp=None, lora=None, layer_idx: int = 0):
        super().__init__()
        assert (tp is None or tp.world == 1) and (cp is None or cp.world == 1) and not lora, "post-norm layers: no tensor / context parallelism, no LoRA"
        self.cfg, self.layer_idx, self.window = cfg, layer_idx, 0
        entry, d = cfg.mixers[layer_idx], cfg.hidden_size
        norm = lambda: nn.Parameter(torch.ones(d, dtype=dtype, device=device))   # noqa: E731
        self.mixer = MIXERS[entry["type"]](cfg.mixer_spec(layer_idx), cfg, dtype, device)
        self.norm1 = norm()
        self.ff = None
        if entry.get("mlp"):
            self.ff = feed_forward(cfg.mlp_spec(layer_idx), cfg, dtype, device)
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
