"""Sequence mixers of models that are described layer by layer, and the parallel layer (mixer and MLP side by side); the layers whose
sublayers run one after the other are in ``post_norm.py`` and ``pre_norm.py``.

A parallel layer computes ``h = norm(x)`` once and adds ``mixer(h) + mlp(h)`` to the residual stream, so all its input projections
read the same rows and both its output projections write the same rows. The layer therefore holds two fused weights:

    in_proj  [mixer projections | gate | MLP up, d]     one product of ``h``; squared ReLU rides on the ``up`` columns
    out_proj [d, mixed | MLP ff]                        one product whose left operand is the [gate | up] range of the first
                                                        product's rows: the mixer writes its gated output over the gate columns

Segments start at multiples of 8 columns (16-byte rows for TMA); padding rows and columns hold zeros. The residual stream is fp32.

Mixers:
  * ``LatentAttentionMixer``: causal attention whose keys and values are decompressed from one normalised latent per token; only
    the latent and a rotated key part shared by the heads are cached. Own softmax scale; queries plain or through a normed latent of their
    own, output gate or none, rotated pairs interleaved or in halves.
  * ``RetentionMixer``: linear attention with one fixed decay per head, a unit-RMS norm per head and a SiLU gate. The state
    [heads, dim, vdim] is fp32.
  * ``GroupedAttentionMixer``: causal attention with fewer key / value heads than query heads, RMS norms per head on queries and keys,
    partial rotation (pairs interleaved or in halves), own scale, keys and values of unequal size; optionally biases, an output gate, keys of
    the query's own chunk of positions or of a sliding window with kept first tokens only, values mixed with those of the first such layer,
    another layer's keys and values in place of own ones, sigmoid weights in place of the soft-max.
  * ``Mamba2LayerMixer``: state-space duality with a short convolution in front and a gated norm in equal parts behind.
  * ``DeltaMixer``: gated delta rule: a linear-attention state that forgets by a decay per token and corrects what it stores under a key.

The modules' ``sequence`` methods are the differentiable PyTorch statement over packed sequences (training, CPU); the generation
engine runs the same weights through ``rl_b200/ops/mixer_ops.py`` (latent attention, retention) and ``rl_b200/ops/sequence_ops.py``.
"""

from __future__ import annotations

import math

import torch
import torch.nn as nn
import torch.nn.functional as TF

from rl_b200.ops import functional as F

from .config import ModelConfig, rotary_table
from .mamba import gated_group_norm, init_decay, ssd_scan


def pad8(n: int) -> int:
    return -(-n // 8) * 8


class DynamicTanh(nn.Module):
    """y = w * tanh(alpha x) + b: a norm without statistics. Evaluated in fp32, returned in ``out_dtype``."""

    def __init__(self, d: int, dtype, device):
        super().__init__()
        self.weight = nn.Parameter(torch.ones(d, dtype=dtype, device=device))
        self.bias = nn.Parameter(torch.zeros(d, dtype=dtype, device=device))
        self.alpha = nn.Parameter(torch.full((), 0.5, dtype=dtype, device=device))

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        y = torch.tanh(self.alpha.float() * x.float()) * self.weight.float() + self.bias.float()
        return y.to(self.weight.dtype)


def rotate_pairs(x: torch.Tensor, positions: torch.Tensor, freq: torch.Tensor, gain: float, interleaved: bool) -> torch.Tensor:
    """fp32 rotation of the leading ``2 * len(freq)`` dimensions of ``x`` [T, H, n]; pairs are (2i, 2i + 1) when ``interleaved``,
    else (i, i + len(freq)). Cosine and sine are multiplied by ``gain``."""
    x = x.float()
    half = freq.numel()
    if half == 0:
        return x
    ang = positions.float()[:, None] * freq[None, :]
    c, s = (ang.cos() * gain)[:, None, :], (ang.sin() * gain)[:, None, :]
    head, rest = x[..., : 2 * half], x[..., 2 * half :]
    u, v = (head[..., 0::2], head[..., 1::2]) if interleaved else (head[..., :half], head[..., half:])
    a, b = u * c - v * s, v * c + u * s
    rot = torch.stack([a, b], dim=-1).flatten(-2) if interleaved else torch.cat([a, b], dim=-1)
    return torch.cat([rot, rest], dim=-1)


class LatentAttentionMixer(nn.Module):
    """Spec, beside the sizes: "q_rank" (queries go through a normed latent of this width), "gate" (output gate, default yes), "interleaved"
    (rotated pairs are (2i, 2i + 1), default yes; else (i, i + dims / 2))."""

    kind = "latent_attention"

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.heads, self.dim, self.rot_dim, self.vdim = spec["heads"], spec["dim"], spec["rot_dim"], spec["vdim"]
        self.rank, self.scale, self.eps = spec["kv_rank"], float(spec["scale"]), cfg.rms_norm_eps
        self.qdim = self.dim + self.rot_dim
        self.latent_width = pad8(self.rank + self.rot_dim)       # row width of the cache: [latent | rotated key | padding]
        H = self.heads
        self.q_rank, self.gate, self.interleaved = spec.get("q_rank", 0), bool(spec.get("gate", True)), bool(spec.get("interleaved", True))
        self.q_off, self.lat_off = 0, pad8(self.q_rank or H * self.qdim)
        self.mix_width = pad8(H * self.vdim)
        end = self.lat_off + pad8(self.rank + self.rot_dim)
        # with a gate the head outputs are written over its columns of the projected rows, else to rows of their own
        self.mix_off, self.in_width = (end, end + self.mix_width) if self.gate else (0, end)
        if self.q_rank:
            self.q_norm = nn.Parameter(torch.ones(self.q_rank, dtype=dtype, device=device))
            self.q_up = nn.Parameter(torch.zeros(pad8(H * self.qdim), pad8(self.q_rank), dtype=dtype, device=device))
        self.kv_norm = nn.Parameter(torch.ones(self.rank, dtype=dtype, device=device))
        self.kv_up = nn.Parameter(torch.empty(H * (self.dim + self.vdim), self.rank, dtype=dtype, device=device))   # [keys | values]
        freq, self.gain = rotary_table(spec["rot"])
        self.register_buffer("freq", freq.to(device), persistent=False)

    def add_projections(self, d: int, dtype, device) -> None:
        """Projections of the mixer's own, in layers that do not fuse them with the MLP's."""
        self.in_proj = nn.Parameter(torch.zeros(self.in_width, d, dtype=dtype, device=device))
        self.out_proj = nn.Parameter(torch.zeros(d, self.mix_width, dtype=dtype, device=device))

    def tensors(self) -> list:
        """(checkpoint leaf, view of a parameter); with projections of the mixer's own."""
        out = [(leaf, self.in_proj[r : r + n]) for leaf, r, n in self.in_rows()]
        out += [(leaf, getattr(self, p) if n is None else getattr(self, p)[r : r + n]) for leaf, p, r, n in self.own_tensors()]
        if self.q_rank:
            out += [("dq.norm", self.q_norm), ("uq", self.q_up[: self.heads * self.qdim, : self.q_rank])]
        return out + [("o", self.out_proj[:, : self.heads * self.vdim])]

    def in_rows(self) -> list:
        """(checkpoint leaf, first row, rows) of this mixer's slices of ``in_proj``."""
        H = self.heads
        out = [("dq", self.q_off, self.q_rank) if self.q_rank else ("q", self.q_off, H * self.qdim), ("dkv", self.lat_off, self.rank + self.rot_dim)]
        return out + ([("g", self.mix_off, H * self.vdim)] if self.gate else [])

    def own_tensors(self) -> list:
        """(checkpoint leaf, parameter name, first row, rows or None)."""
        H = self.heads
        return [("dkv.norm", "kv_norm", 0, None), ("uk", "kv_up", 0, H * self.dim), ("uv", "kv_up", H * self.dim, H * self.vdim)]

    def key_parts(self, p: torch.Tensor, positions: torch.Tensor):
        """From the projected rows: normalised latent [T, rank] and rotated shared key [T, rot_dim], both fp32."""
        lat = p[:, self.lat_off : self.lat_off + self.rank].float()
        lat = lat * torch.rsqrt(lat.pow(2).mean(-1, keepdim=True) + self.eps) * self.kv_norm.float()
        kr = p[:, self.lat_off + self.rank : self.lat_off + self.rank + self.rot_dim]
        return lat, rotate_pairs(kr[:, None], positions, self.freq, self.gain, self.interleaved)[:, 0]

    def project_queries(self, p: torch.Tensor) -> torch.Tensor:
        """Rows with the queries from column ``q_off`` on: the projected rows, or the product of the normed query latent."""
        if not self.q_rank:
            return p
        c = rms_unit(p[:, : self.q_rank].float(), self.eps) * self.q_norm.float()
        return _linear(TF.pad(c, (0, self.q_up.shape[1] - self.q_rank)).to(p.dtype), self.q_up)

    def queries(self, p: torch.Tensor, positions: torch.Tensor):
        q = p[:, self.q_off : self.q_off + self.heads * self.qdim].reshape(-1, self.heads, self.qdim)
        return torch.cat([q[..., : self.dim].float(), rotate_pairs(q[..., self.dim :], positions, self.freq, self.gain, self.interleaved)], dim=-1)

    def sequence(self, p: torch.Tensor, positions: torch.Tensor, cu_seqlens: torch.Tensor) -> torch.Tensor:
        """Head outputs [T, heads * vdim] of packed whole sequences, gated where the mixer has a gate."""
        T, H = p.shape[0], self.heads
        lat, kr = self.key_parts(p, positions)
        lat = lat.to(p.dtype)
        k = TF.linear(lat, self.kv_up[: H * self.dim]).reshape(T, H, self.dim)
        v = TF.linear(lat, self.kv_up[H * self.dim :]).reshape(T, H, self.vdim).float()
        k = torch.cat([k.float(), kr[:, None].expand(T, H, self.rot_dim)], dim=-1)
        q = self.queries(self.project_queries(p), positions)
        out = []
        cu = cu_seqlens.tolist()
        for s, e in zip(cu[:-1], cu[1:]):
            z = torch.einsum("ihd,jhd->hij", q[s:e], k[s:e]) * self.scale
            z = z.masked_fill(torch.ones(e - s, e - s, dtype=torch.bool, device=z.device).triu(1), float("-inf"))
            out.append(torch.einsum("hij,jhd->ihd", torch.softmax(z, -1), v[s:e]))
        y = torch.cat(out).reshape(T, H * self.vdim)
        if not self.gate:
            return y.to(p.dtype)
        return (y * torch.sigmoid(p[:, self.mix_off : self.mix_off + H * self.vdim].float())).to(p.dtype)


class RetentionMixer(nn.Module):
    kind = "retention"

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.heads, self.dim, self.vdim, self.eps = spec["heads"], spec["dim"], spec["vdim"], cfg.rms_norm_eps
        H = self.heads
        self.q_off = 0
        self.k_off = pad8(H * self.dim)
        self.v_off = self.k_off + pad8(H * self.dim)
        self.mix_off = self.v_off + pad8(H * self.vdim)
        self.mix_width = pad8(H * self.vdim)
        self.in_width = self.mix_off + self.mix_width
        freq, self.gain = rotary_table(spec["rot"])
        self.register_buffer("freq", freq.to(device), persistent=False)
        self.register_buffer("decay", torch.tensor(spec["decay"], dtype=torch.float32, device=device), persistent=False)
        # log2 of the decays from the configuration's own precision: powers of a decay are taken as exp2(n * log2 decay)
        self.register_buffer("log2_decay", torch.tensor(spec["decay"], dtype=torch.float64).log2().clamp(min=-1e4).float().to(device), persistent=False)

    def in_rows(self) -> list:
        H = self.heads
        return [("q", self.q_off, H * self.dim), ("k", self.k_off, H * self.dim), ("v", self.v_off, H * self.vdim), ("g", self.mix_off, H * self.vdim)]

    def own_tensors(self) -> list:
        return []

    def qkv(self, p: torch.Tensor, positions: torch.Tensor):
        """fp32 rotated queries, rotated and scaled keys [T, H, dim], values [T, H, vdim]."""
        H = self.heads
        q = rotate_pairs(p[:, self.q_off : self.q_off + H * self.dim].reshape(-1, H, self.dim), positions, self.freq, self.gain, False)
        k = rotate_pairs(p[:, self.k_off : self.k_off + H * self.dim].reshape(-1, H, self.dim), positions, self.freq, self.gain, False)
        v = p[:, self.v_off : self.v_off + H * self.vdim].reshape(-1, H, self.vdim).float()
        return q, k * self.dim ** -0.5, v

    def finish(self, o: torch.Tensor, p: torch.Tensor) -> torch.Tensor:
        """Unit-RMS norm per head and SiLU gate of the head outputs ``o`` [T, H, vdim] (fp32)."""
        H = self.heads
        o = o * torch.rsqrt(o.pow(2).mean(-1, keepdim=True) + self.eps)
        g = p[:, self.mix_off : self.mix_off + H * self.vdim].float()
        return (o.reshape(-1, H * self.vdim) * TF.silu(g)).to(p.dtype)

    def scan(self, q, k, v, S, chunk: int = 64):
        """Outputs [L, H, vdim] of one sequence (piece) starting from state ``S`` [H, dim, vdim], and the state it leaves. Chunk by
        chunk: the products inside a chunk are one masked score matrix, only chunk borders are visited one after the other."""
        outs = []
        ld = self.log2_decay.to(q.dtype)
        for s in range(0, q.shape[0], chunk):
            qc, kc, vc = q[s : s + chunk], k[s : s + chunk], v[s : s + chunk]
            n = qc.shape[0]
            i = torch.arange(n, device=q.device)
            gap = (i[:, None] - i[None, :]).to(q.dtype)
            w = torch.where(gap >= 0, torch.exp2(gap.clamp(min=0) * ld[:, None, None]), torch.zeros((), device=q.device, dtype=q.dtype))
            o = torch.einsum("hij,jhv->ihv", torch.einsum("ihd,jhd->hij", qc, kc) * w, vc)
            o = o + torch.einsum("ihd,hdv->ihv", qc, S) * torch.exp2((i + 1)[:, None].to(q.dtype) * ld)[..., None]
            tail = torch.exp2((n - 1 - i)[:, None].to(q.dtype) * ld)
            S = S * torch.exp2(n * ld)[:, None, None] + torch.einsum("jhd,jhv->hdv", kc * tail[..., None], vc)
            outs.append(o)
        return torch.cat(outs), S

    def sequence(self, p: torch.Tensor, positions: torch.Tensor, cu_seqlens: torch.Tensor) -> torch.Tensor:
        q, k, v = self.qkv(p, positions)
        cu = cu_seqlens.tolist()
        zero = torch.zeros(self.heads, self.dim, self.vdim, dtype=torch.float32, device=p.device)
        return self.finish(torch.cat([self.scan(q[s:e], k[s:e], v[s:e], zero)[0] for s, e in zip(cu[:-1], cu[1:])]), p)


def rms_unit(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


class GroupedAttentionMixer(nn.Module):
    """Spec, beside the sizes:
      "bias"         biases on the projections (default yes)
      "qk_norm"      RMS norms per head on queries and keys (default yes)
      "interleaved"  rotated pairs are (2i, 2i + 1) (default yes); else (i, i + dims / 2)
      "mask"         with "mask_kind" "chunk" (default) {"size"}: position i sees j <= i of the same run of ``size`` positions, counted from the
                     sequence's first; with "window" {"size", "keep_first"}: it sees j <= i with i - j < size or j < keep_first
      "weights"      "softmax" (default), or "sigmoid": every visible key weighs sigmoid(score + a number per head), unnormalised
      "gate"         the head outputs are multiplied by sigmoid of a projection of the mixer's input (default no)
      "v_mix"        values become (1 - share) v + share v_first with v_first the first such layer's
      "kv_from"      index of the layer whose keys and values are read; the layer projects none of its own"""

    kind = "attention"

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
        self.scale, self.eps = float(spec["scale"]), cfg.rms_norm_eps
        self.kv_from = spec.get("kv_from")
        self.gate, self.sigmoid = bool(spec.get("gate")), spec.get("weights", "softmax") == "sigmoid"
        self.q_off, end = 0, pad8(self.heads * self.dim)
        self.k_off = self.v_off = end
        if self.kv_from is None:
            self.v_off = self.k_off + pad8(self.kv_heads * self.dim)
            end = self.v_off + pad8(self.kv_heads * self.vdim)
        self.mix_width = pad8(self.heads * self.vdim)
        # with a gate the head outputs are written over its columns of the projected rows, else to rows of their own
        self.mix_off, self.in_width = (end, end + self.mix_width) if self.gate else (0, end)
        d = cfg.hidden_size
        self.in_proj = nn.Parameter(torch.zeros(self.in_width, d, dtype=dtype, device=device))
        self.out_proj = nn.Parameter(torch.zeros(d, self.mix_width, dtype=dtype, device=device))
        self.in_bias = self.out_bias = None
        if spec.get("bias", True):
            self.in_bias = nn.Parameter(torch.zeros(self.in_width, dtype=dtype, device=device))
            self.out_bias = nn.Parameter(torch.zeros(d, dtype=dtype, device=device))
        self.interleaved, mask = bool(spec.get("interleaved", True)), spec.get("mask")
        windowed = spec.get("mask_kind", "chunk") == "window"
        self.chunk = int(mask["size"]) if mask and not windowed else 0
        self.window, self.keep = (int(mask["size"]), int(mask.get("keep_first", 0))) if mask and windowed else (0, 0)
        self.v_mix = bool(spec.get("v_mix"))
        if self.v_mix:
            self.v_share = nn.Parameter(torch.full((), 0.5, dtype=dtype, device=device))
        self.qk_norm = bool(spec.get("qk_norm", True))
        self.q_norm = self.k_norm = self.offset = None
        if self.qk_norm:
            self.q_norm = nn.Parameter(torch.ones(self.dim, dtype=dtype, device=device))
            self.k_norm = nn.Parameter(torch.ones(self.dim, dtype=dtype, device=device))
        if self.sigmoid:       # added to the scores; starts where as many keys as the mask shows weigh about one together
            self.offset = nn.Parameter(torch.full((self.heads,), -math.log(self.window or self.chunk or 1024), dtype=dtype, device=device))
        freq, self.gain = rotary_table(spec["rot"])
        self.register_buffer("freq", freq.to(device), persistent=False)

    def tensors(self) -> list:
        """(checkpoint leaf, view of a parameter)."""
        own = self.kv_from is None
        rows = [("q", self.q_off, self.heads * self.dim)]
        if own:
            rows += [("k", self.k_off, self.kv_heads * self.dim), ("v", self.v_off, self.kv_heads * self.vdim)]
        if self.gate:
            rows.append(("g", self.mix_off, self.heads * self.vdim))
        out = []
        for leaf, r, n in rows:
            out += [(leaf, self.in_proj[r : r + n])] + ([(leaf + ".b", self.in_bias[r : r + n])] if self.in_bias is not None else [])
        if self.qk_norm:
            out += [("q.norm", self.q_norm)] + ([("k.norm", self.k_norm)] if own else [])
        if self.sigmoid:
            out.append(("pb", self.offset))
        out.append(("o", self.out_proj[:, : self.heads * self.vdim]))
        return out + ([("o.b", self.out_bias)] if self.out_bias is not None else []) + ([("vmix", self.v_share)] if self.v_mix else [])

    def values(self, p: torch.Tensor) -> torch.Tensor:
        """The layer's own values, columns of the projected rows."""
        return p[:, self.v_off : self.v_off + self.kv_heads * self.vdim]

    def _prepared(self, x: torch.Tensor, norm, positions: torch.Tensor) -> torch.Tensor:
        x = x.float()
        if self.qk_norm:
            x = rms_unit(x, self.eps) * norm.float()
        return rotate_pairs(x, positions, self.freq, self.gain, self.interleaved)

    def queries(self, p: torch.Tensor, positions: torch.Tensor) -> torch.Tensor:
        """fp32 normed and rotated queries [T, heads, dim]."""
        return self._prepared(p[:, self.q_off : self.q_off + self.heads * self.dim].reshape(-1, self.heads, self.dim), self.q_norm, positions)

    def keys_values(self, p: torch.Tensor, positions: torch.Tensor, first=None):
        """fp32 normed and rotated keys [T, kv_heads, dim], values [T, kv_heads, vdim] (mixed with ``first``)."""
        v = self.values(p).float()
        if first is not None:
            v = (1 - self.v_share.float()) * v + self.v_share.float() * first.float()
        k = self._prepared(p[:, self.k_off : self.k_off + self.kv_heads * self.dim].reshape(-1, self.kv_heads, self.dim), self.k_norm, positions)
        return k, v.reshape(-1, self.kv_heads, self.vdim)

    def qkv(self, p: torch.Tensor, positions: torch.Tensor, first=None):
        return (self.queries(p, positions), *self.keys_values(p, positions, first))

    def hidden(self, i: torch.Tensor, j: torch.Tensor) -> torch.Tensor:
        """Whether position i does not see position j (tensors that broadcast)."""
        h = j > i
        if self.chunk:
            h = h | (i // self.chunk != j // self.chunk)
        if self.window:
            h = h | ((i - j >= self.window) & (j >= self.keep))
        return h

    def weigh(self, z: torch.Tensor, hidden: torch.Tensor) -> torch.Tensor:
        """Weights of the keys from scaled scores [..., heads, queries, keys]."""
        if self.sigmoid:
            return torch.sigmoid(z + self.offset.float()[:, None, None]).masked_fill(hidden, 0.0)
        return torch.softmax(z.masked_fill(hidden, float("-inf")), -1)

    def gated(self, y: torch.Tensor, p: torch.Tensor) -> torch.Tensor:
        """Head outputs [T, heads * vdim] behind the output gate where there is one."""
        return y * torch.sigmoid(p[:, self.mix_off : self.mix_off + self.heads * self.vdim].float()) if self.gate else y

    def sequence(self, p: torch.Tensor, positions: torch.Tensor, cu_seqlens: torch.Tensor, first=None, kv=None) -> torch.Tensor:
        """Head outputs [T, heads * vdim] of packed whole sequences. ``kv``: prepared keys and values (None: the layer's own)."""
        q = self.queries(p, positions)
        k, v = self.keys_values(p, positions, first) if kv is None else kv
        n = self.heads // self.kv_heads
        k, v = k.repeat_interleave(n, dim=1), v.repeat_interleave(n, dim=1)
        out = []
        cu = cu_seqlens.tolist()
        for s, e in zip(cu[:-1], cu[1:]):
            z = torch.einsum("ihd,jhd->hij", q[s:e], k[s:e]) * self.scale
            t = torch.arange(e - s, device=z.device)
            out.append(torch.einsum("hij,jhd->ihd", self.weigh(z, self.hidden(t[:, None], t[None, :])), v[s:e]))
        return self.gated(torch.cat(out).reshape(-1, self.heads * self.vdim), p).to(p.dtype)


class RecurrentMixer(nn.Module):
    """What the mixers with a short convolution and a state per sequence share: the convolved channels are one column range of the
    projected rows, [conv_off, conv_off + channels), and the state is [heads, dim, vdim] in fp32."""

    in_bias = out_bias = None

    def piece_bounds(self, cu_seqlens: torch.Tensor) -> list:
        cu = cu_seqlens.tolist()
        return list(zip(cu[:-1], cu[1:]))

    def convolve(self, x: torch.Tensor, before: torch.Tensor) -> torch.Tensor:
        """silu of the causal convolution of one sequence piece's rows [L, channels]; ``before`` [taps - 1, channels] stood in front."""
        L, n = x.shape[0], self.taps
        xp = torch.cat([before.to(x.dtype), x]).float()
        y = sum(xp[j : j + L] * self.conv[:, j].float() for j in range(n))
        if self.conv_bias is not None:
            y = y + self.conv_bias.float()
        return TF.silu(y).to(x.dtype)

    def sequence(self, p: torch.Tensor, positions: torch.Tensor, cu_seqlens: torch.Tensor) -> torch.Tensor:
        """Mixer outputs (before the output product) of packed whole sequences."""
        out = []
        for s, e in self.piece_bounds(cu_seqlens):
            u = self.convolve(p[s:e, self.conv_off : self.conv_off + self.channels], p.new_zeros(self.taps - 1, self.channels))
            zero = torch.zeros(self.heads, self.dim, self.vdim, dtype=torch.float32, device=p.device)
            out.append(self.finish(self.scan(u, p[s:e], zero)[0], p[s:e]))
        return torch.cat(out)


class Mamba2LayerMixer(RecurrentMixer):
    """S <- exp(-exp(A_log) dt) S + dt B x^T, y = S^T C + D x per head; dt = softplus(projection + dt_bias). Heads in equal runs share a
    group's B and C. ``dim`` is the state width."""

    kind = "mamba2"

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.heads, self.vdim, self.dim, self.groups = spec["heads"], spec["vdim"], spec["state"], spec["groups"]
        self.norm_groups, self.taps, self.eps = spec["norm_groups"], spec["conv"], cfg.rms_norm_eps
        self.inner = self.heads * self.vdim
        self.channels = self.inner + 2 * self.groups * self.dim
        self.z_off, self.conv_off, self.dt_off = 0, self.inner, self.inner + self.channels      # (one checkpoint tensor: no padding between)
        self.in_width, self.mix_width = pad8(self.dt_off + self.heads), pad8(self.inner)
        P = lambda *shape: nn.Parameter(torch.zeros(*shape, dtype=dtype, device=device))   # noqa: E731
        self.in_proj, self.out_proj = P(self.in_width, cfg.hidden_size), P(cfg.hidden_size, self.mix_width)
        self.conv, self.conv_bias = P(self.channels, self.taps), P(self.channels)
        self.A_log, self.dt_bias, self.D = P(self.heads), P(self.heads), nn.Parameter(torch.ones(self.heads, dtype=dtype, device=device))
        self.norm = nn.Parameter(torch.ones(self.inner, dtype=dtype, device=device))

    def tensors(self) -> list:
        return [("in", self.in_proj[: self.dt_off + self.heads]), ("conv", self.conv),
                ("conv.b", self.conv_bias), ("dt_bias", self.dt_bias), ("A_log", self.A_log), ("D", self.D), ("norm", self.norm), ("o", self.out_proj[:, : self.inner])]

    def reset_special(self, gen: torch.Generator) -> None:
        init_decay(self.A_log, self.dt_bias, gen)

    def parts(self, u: torch.Tensor, p: torch.Tensor):
        """fp32 x [T, heads, vdim], B and C [T, groups, dim], step sizes and log decays [T, heads]."""
        u, n = u.float(), self.groups * self.dim
        dt = TF.softplus(p[:, self.dt_off : self.dt_off + self.heads].float() + self.dt_bias.float())
        return (u[:, : self.inner].reshape(-1, self.heads, self.vdim), u[:, self.inner : self.inner + n].reshape(-1, self.groups, self.dim),
                u[:, self.inner + n :].reshape(-1, self.groups, self.dim), dt, -self.A_log.float().exp() * dt)

    def scan(self, u: torch.Tensor, p: torch.Tensor, S: torch.Tensor, chunk: int = 64):
        """(outputs [L, heads, vdim], state left) of one piece that starts from state ``S`` [heads, dim, vdim]."""
        x, B, C, dt, _ = self.parts(u, p)
        y, S = ssd_scan(x[None], dt[None], -self.A_log.float().exp(), B[None], C[None], chunk, S.transpose(1, 2)[None])
        return y[0] + self.D.float()[:, None] * x, S[0].transpose(1, 2)

    def finish(self, y: torch.Tensor, p: torch.Tensor) -> torch.Tensor:
        return gated_group_norm(y.reshape(-1, self.inner), p[:, self.z_off : self.z_off + self.inner], self.norm, self.norm_groups, self.eps)


class DeltaMixer(RecurrentMixer):
    """S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q per head, with unit keys and queries, beta = sigmoid(W_b h) and
    g = exp(-exp(A_log) softplus(W_a h + dt_bias)); then an RMS norm per head and a SiLU gate."""

    kind = "delta"
    conv_bias = None
    unit_eps = 1e-6        # under the root of the unit norms of queries and keys

    def __init__(self, spec: dict, cfg: ModelConfig, dtype, device):
        super().__init__()
        self.heads, self.kv_heads, self.dim, self.vdim = spec["heads"], spec["kv_heads"], spec["dim"], spec["vdim"]
        self.taps, self.eps = spec["conv"], cfg.rms_norm_eps
        H, n = self.heads, self.kv_heads * self.dim
        self.channels, self.conv_off = 2 * n + H * self.vdim, 0
        self.g_off = pad8(self.channels)
        self.b_off = self.g_off + pad8(H * self.vdim)
        self.a_off = self.b_off + pad8(H)
        self.in_width, self.mix_width = self.a_off + pad8(H), pad8(H * self.vdim)
        P = lambda *shape: nn.Parameter(torch.zeros(*shape, dtype=dtype, device=device))   # noqa: E731
        self.in_proj, self.out_proj = P(self.in_width, cfg.hidden_size), P(cfg.hidden_size, self.mix_width)
        self.conv = P(self.channels, self.taps)
        self.A_log, self.dt_bias = P(H), P(H)
        self.norm = nn.Parameter(torch.ones(self.vdim, dtype=dtype, device=device))

    def tensors(self) -> list:
        H, n, hv = self.heads, self.kv_heads * self.dim, self.heads * self.vdim
        out = []
        for leaf, r, k in (("q", 0, n), ("k", n, n), ("v", 2 * n, hv)):
            out += [(leaf, self.in_proj[r : r + k]), (leaf + ".conv", self.conv[r : r + k])]
        out += [(leaf, self.in_proj[r : r + k]) for leaf, r, k in (("g", self.g_off, hv), ("b", self.b_off, H), ("a", self.a_off, H))]
        return out + [("A_log", self.A_log), ("dt_bias", self.dt_bias), ("norm", self.norm), ("o", self.out_proj[:, :hv])]

    def reset_special(self, gen: torch.Generator) -> None:
        init_decay(self.A_log, self.dt_bias, gen)

    def parts(self, u: torch.Tensor, p: torch.Tensor):
        """fp32 unit queries (scaled by dim^-1/2) and keys [T, heads, dim], values, step sizes beta and log decays [T, heads]."""
        u, n, H = u.float(), self.kv_heads * self.dim, self.heads
        q, k = (t.reshape(-1, self.kv_heads, self.dim) for t in (u[:, :n], u[:, n : 2 * n]))
        q, k = (t * torch.rsqrt(t.pow(2).sum(-1, keepdim=True) + self.unit_eps) for t in (q, k))
        rep = H // self.kv_heads
        beta = torch.sigmoid(p[:, self.b_off : self.b_off + H].float())
        lg = -self.A_log.float().exp() * TF.softplus(p[:, self.a_off : self.a_off + H].float() + self.dt_bias.float())
        return (q.repeat_interleave(rep, 1) * self.dim ** -0.5, k.repeat_interleave(rep, 1), u[:, 2 * n :].reshape(-1, H, self.vdim), beta, lg)

    def scan(self, u: torch.Tensor, p: torch.Tensor, S: torch.Tensor, chunk: int = 64):
        """(outputs [L, heads, vdim], state left) of one piece. Inside a chunk with start state S the writes U solve the unit lower
        triangular system (I + A) U = beta (V - decay K S), A_ij = beta_i decay_i / decay_j k_i . k_j for j < i."""
        outs = []
        q, k, v, beta, lg = (t.transpose(0, 1) for t in self.parts(u, p))          # [heads, L, ...]
        for s in range(0, q.shape[1], chunk):
            qc, kc, vc, bc = q[:, s : s + chunk], k[:, s : s + chunk], v[:, s : s + chunk], beta[:, s : s + chunk, None]
            cum = lg[:, s : s + chunk].cumsum(-1)
            n = qc.shape[1]
            low = torch.ones(n, n, dtype=torch.bool, device=q.device).tril()
            ratio = torch.where(low, cum[:, :, None] - cum[:, None, :], torch.full((), float("-inf"), device=q.device)).exp()
            A = (bc * ratio * (kc @ kc.transpose(1, 2))).tril(-1)
            eye = torch.eye(n, device=q.device)
            U = torch.linalg.solve_triangular(eye + A, bc * (vc - cum.exp()[..., None] * (kc @ S)), upper=False, unitriangular=True)
            outs.append(cum.exp()[..., None] * (qc @ S) + (ratio * (qc @ kc.transpose(1, 2))) @ U)
            end = cum[:, -1:]
            S = end.exp()[..., None] * S + (kc * (end - cum).exp()[..., None]).transpose(1, 2) @ U
        return torch.cat(outs, 1).transpose(0, 1), S

    def finish(self, o: torch.Tensor, p: torch.Tensor) -> torch.Tensor:
        hv = self.heads * self.vdim
        y = (rms_unit(o, self.eps) * self.norm.float()).reshape(-1, hv)
        return (y * TF.silu(p[:, self.g_off : self.g_off + hv].float())).to(p.dtype)


MIXERS = {m.kind: m for m in (LatentAttentionMixer, RetentionMixer, GroupedAttentionMixer, Mamba2LayerMixer, DeltaMixer)}


class ParallelBlock(nn.Module):
    """x <- x + mixer(norm(x)) + mlp(norm(x)); the MLP may be absent."""

    def __init__(self, cfg: ModelConfig, dtype, device, tp=None, ep=None, cp=None, lora=None, layer_idx: int = 0):
        super().__init__()
        assert (tp is None or tp.world == 1) and (cp is None or cp.world == 1) and not lora, \
            "parallel mixer layers: no tensor / context parallelism, no LoRA"
        self.cfg, self.layer_idx, self.window = cfg, layer_idx, 0
        entry = cfg.mixers[layer_idx]
        d = cfg.hidden_size
        self.norm = DynamicTanh(d, dtype, device)
        self.mixer = MIXERS[entry["type"]](cfg.mixer_spec(layer_idx), cfg, dtype, device)
        self.ff = entry["mlp"]["ff"] if entry.get("mlp") else 0
        self.up_off = self.mixer.in_width                  # first MLP column of the projected rows; squared ReLU from here on
        self.in_width = self.up_off + pad8(self.ff)
        self.out_width = self.mixer.mix_width + pad8(self.ff)
        self.in_proj = nn.Parameter(torch.zeros(self.in_width, d, dtype=dtype, device=device))
        self.out_proj = nn.Parameter(torch.zeros(d, self.out_width, dtype=dtype, device=device))
        self.self_attn = self.mlp = None                   # (the names other families' walkers look for)

    def tensor_views(self, prefix: str) -> list:
        """(checkpoint name, view of a parameter) of every tensor of this layer."""
        m = self.mixer
        out = [(f"{prefix}norm1", self.norm.weight), (f"{prefix}norm1.b", self.norm.bias), (f"{prefix}norm1.alpha", self.norm.alpha)]
        out += [(f"{prefix}mix.{leaf}", self.in_proj[r : r + n]) for leaf, r, n in m.in_rows()]
        for leaf, pname, r, n in m.own_tensors():
            p = getattr(m, pname)
            out.append((f"{prefix}mix.{leaf}", p if n is None else p[r : r + n]))
        out.append((f"{prefix}mix.o", self.out_proj[:, : m.heads * m.vdim]))
        if self.ff:
            out += [(f"{prefix}mlp.up", self.in_proj[self.up_off : self.up_off + self.ff]),
                    (f"{prefix}mlp.down", self.out_proj[:, m.mix_width : m.mix_width + self.ff])]
        return out

    def forward(self, x, positions, inv_freq, cu_seqlens, max_seqlen):
        h = self.norm(x)
        p = _linear(h, self.in_proj)
        parts = [TF.pad(self.mixer.sequence(p, positions, cu_seqlens), (0, self.mixer.mix_width - self.mixer.heads * self.mixer.vdim))]
        if self.ff:
            parts.append(F.plain_act(p[:, self.up_off :].float(), "relu2").to(p.dtype))
        return x + _linear(torch.cat(parts, dim=1), self.out_proj).float()


def _linear(x: torch.Tensor, w: torch.Tensor) -> torch.Tensor:
    """The framework's GEMM where its kernels take the shape and type; otherwise the library's."""
    if x.dtype == torch.bfloat16 and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0:
        return F.linear(x, w)
    return TF.linear(x, w)
