"""The layer whose sublayers run one after the other on norms of the residual stream:

    x <- x + mixer(norm1(x));   x <- x + feed-forward(norm2(x))

With norms on both sides ("both") what a sublayer returns is normed too, and with a layer scale multiplied element by element:

    x <- x + ls1 norm1b(mixer(norm1(x)));   x <- x + ls2 norm2b(feed-forward(norm2(x)))

With a token shift the mixer reads h + (h' - h) s in place of h = norm1(x), element by element, h' being the h of the sequence's token before
(zeros for the first). The feed-forward (``gated.py``) may be absent. The residual stream and the norms are fp32. Attention layers may take over
a share of an earlier layer's values (``GroupedAttentionMixer.v_mix``): the first of them hands its values on to the others; or read another
layer's keys and values (``kv_from``).

The modules' ``forward`` methods are the differentiable PyTorch statement (training, CPU); the generation engine runs the same weights
through ``rl_b200/ops/mixer_ops.py``, ``sequence_ops.py`` and ``layer_ops.py``.
"""

from __future__ import annotations

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
        self.norm1b = self.norm2b = self.ls1 = self.ls2 = self.shift = None
        if cfg.norm_place == "both":
            self.norm1b, self.norm2b = norm(), norm() if self.ff is not None else None
        if cfg.layer_scale:
            self.ls1, self.ls2 = norm(), norm() if self.ff is not None else None
        if cfg.token_shift:
            self.shift = nn.Parameter(torch.full((d,), 0.5, dtype=dtype, device=device))
        # whether a later layer reads this one's keys and values
        self.lends = any(e["mixer"].get("kv_from") == layer_idx for e in cfg.mixers)
        self.self_attn = self.mlp = None                   # (the names other families' walkers look for)

    def tensor_views(self, prefix: str) -> list:
        """(checkpoint name, view of a parameter) of every tensor of this layer."""
        out = [(f"{prefix}norm1", self.norm1)] + [(f"{prefix}mix.{leaf}", t) for leaf, t in self.mixer.tensors()]
        if self.ff is not None:
            out += [(f"{prefix}norm2", self.norm2)] + [(f"{prefix}mlp.{leaf}", t) for leaf, t in self.ff.tensors()]
        return out + [(f"{prefix}{n}", getattr(self, n)) for n in ("norm1b", "norm2b", "ls1", "ls2", "shift") if getattr(self, n) is not None]

    def normed(self, x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
        return (rms_unit(x, self.cfg.rms_norm_eps) * w.float()).to(w.dtype)

    def shifted(self, h: torch.Tensor, cu_seqlens: torch.Tensor) -> torch.Tensor:
        if self.shift is None:
            return h
        first = torch.zeros(h.shape[0], dtype=torch.bool, device=h.device)
        starts = cu_seqlens[:-1].long()
        first[starts[starts < h.shape[0]]] = True
        before = torch.cat([h[:1], h[:-1]]).float().masked_fill(first[:, None], 0.0)
        return (h.float() + (before - h.float()) * self.shift.float()).to(h.dtype)

    def joined(self, x: torch.Tensor, y: torch.Tensor, norm, scale) -> torch.Tensor:
        y = y.float()
        if norm is not None:
            y = rms_unit(y, self.cfg.rms_norm_eps) * norm.float()
        return x + (y if scale is None else y * scale.float())

    def forward(self, x, positions, handed: dict, cu_seqlens, max_seqlen):
        """``handed``: what earlier layers hand on: "values" [T, kv_heads * vdim] of the first layer that mixes them, and by layer index the prepared
        keys and values of layers that lend them. Returns (x, the same for the next layer)."""
        m, values = self.mixer, handed.get("values")
        p = _linear(self.shifted(self.normed(x, self.norm1), cu_seqlens), m.in_proj)
        if m.kind == "attention":
            kv = handed[m.kv_from] if m.kv_from is not None else None
            if self.lends:
                kv = m.keys_values(p, positions, values if m.v_mix else None)
                handed = handed | {self.layer_idx: kv}
            y = m.sequence(p, positions, cu_seqlens, values if m.v_mix else None, kv)
            if m.v_mix and values is None:
                handed = handed | {"values": m.values(p)}
        else:
            y = m.sequence(p, positions, cu_seqlens)
        x = self.joined(x, _linear(TF.pad(y, (0, m.mix_width - y.shape[1])), m.out_proj), self.norm1b, self.ls1)
        if self.ff is not None:
            x = self.joined(x, self.ff(self.normed(x, self.norm2)), self.norm2b, self.ls2)
        return x, handed
