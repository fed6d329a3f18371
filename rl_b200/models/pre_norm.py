"""The layer whose sublayers run one after the other on norms of the residual stream:

    x <- x + mixer(norm1(x));   x <- x + feed-forward(norm2(x))

The feed-forward (``gated.py``) may be absent. The residual stream and the norms are fp32. Attention layers may take over a share of an
earlier layer's values (``GroupedAttentionMixer.v_mix``): the first of them hands its values on to the others.

The modules' ``forward`` methods are the differentiable PyTorch statement (training, CPU); the generation engine runs the same weights
through ``rl_b200/ops/mixer_ops.py``, ``sequence_ops.py`` and ``layer_ops.py``.
"""

from __future__ import annotations

from typing import Optional

import torch
import torch.nn as nn
import torch.nn.functional as TF

from .config import ModelConfig
from .gated import feed_forward
from .mixers import MIXERS, _linear, rms_unit


class PreNormBlock(nn.Module):
    def __init__(self, cfg: ModelConfig, dtype, device, tp=None, ep=None, cp=None, lora=None, layer_idx: int = 0):
        super().__init__()
        assert (tp is None or tp.world == 1) and (cp is None or cp.world == 1) and not lora, "pre-norm mixer layers: no tensor / context parallelism, no LoRA"
        self.cfg, self.layer_idx, self.window = cfg, layer_idx, 0
        entry, d = cfg.mixers[layer_idx], cfg.hidden_size
        norm = lambda: nn.Parameter(torch.ones(d, dtype=dtype, device=device))   # noqa: E731
        self.mixer = MIXERS[entry["type"]](cfg.mixer_spec(layer_idx), cfg, dtype, device)
        if not hasattr(self.mixer, "in_proj"):
            self.mixer.add_projections(d, dtype, device)
        self.norm1 = norm()
        self.ff = None
        if entry.get("mlp"):
            self.ff = feed_forward(cfg.mlp_spec(layer_idx), cfg, dtype, device)
            self.norm2 = norm()
        self.self_attn = self.mlp = None                   # (the names other families' walkers look for)

    def tensor_views(self, prefix: str) -> list:
        """(checkpoint name, view of a parameter) of every tensor of this layer."""
        out = [(f"{prefix}norm1", self.norm1)] + [(f"{prefix}mix.{leaf}", t) for leaf, t in self.mixer.tensors()]
        if self.ff is not None:
            out += [(f"{prefix}norm2", self.norm2)] + [(f"{prefix}mlp.{leaf}", t) for leaf, t in self.ff.tensors()]
        return out

    def normed(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        return (rms_unit(x, self.cfg.rms_norm_eps) * w.float()).to(w.dtype)

    def forward(self, x, positions, values: Optional[torch.Tensor], cu_seqlens, max_seqlen):
        """``values`` [T, kv_heads * vdim]: those of the first layer that mixes them, None before it. Returns (x, values)."""
        m = self.mixer
        p = _linear(self.normed(x, self.norm1), m.in_proj)
        if m.kind == "attention":
            y = m.sequence(p, positions, cu_seqlens, values if m.v_mix else None)
            if m.v_mix and values is None:
                values = m.values(p)
        else:
            y = m.sequence(p, positions, cu_seqlens)
        x = x + _linear(TF.pad(y, (0, m.mix_width - y.shape[1])), m.out_proj).float()
        if self.ff is not None:
            x = x + self.ff(self.normed(x, self.norm2)).float()
        return x, values
