"""Operators of parallel mixer layers (``rl_b200/models/mixers.py``) in the generation engine, over a batch of token rows that mixes
single decoded tokens and portions of prompts.

Each operator has the native sm_100a body (CUDA tensors, bf16 or fp32) and a plain PyTorch statement (CPU tensors). A layer is

    p = in_proj(h)               fused projection, squared ReLU on the MLP columns (epilogue)
    latent_* / retention_*       the mixer; writes its gated output over the gate columns of ``p``
    h = out_proj_(x, p)          x += p[gate | up] @ out_proj^T, the loop's additions and the NEXT layer's dynamic-tanh norm (epilogue)

so nothing but the two products and the mixer touches memory. fp32 models run every product in true fp32.
"""

from __future__ import annotations

from dataclasses import dataclass
from typing import Optional

import torch

from . import lib as _L
from .lib import F as CF
from .lib import I, L as LL, P, call, ptr, register, stream_ptr, use_native

register("rlb_embed_rows", [P, I, P, I, P, P, P, P, P, P, P, LL, I, I, CF, P, P])
register("rlb_gemm_rows", [P, P, P, I, I, I, LL, LL, LL, I, I, I, P, LL, P, P, P, P, P, P])
register("rlb_latent_prep", [P, I, LL, LL, I, I, I, I, I, I, I, I, I, P, P, P, P, I, CF, CF, P, P, P])
register("rlb_latent_rows", [P, I, I, LL, I, I, I, I, I, I, I, I, I, I, P, P, I, P, P, CF, P, P])
register("rlb_retention_rows", [P, I, I, I, LL, I, I, I, I, I, I, I, P, P, P, P, LL, P, P, I, CF, CF, CF, P, P])

NO_ACT = 1 << 30


@dataclass
class TokenBatch:
    """Rows of one engine step, single tokens first, then portions in order of length.

    Rows [0, n_single) are one token each of as many sequences; rows [n_single, T) are portions (``cu`` [n + 1], row offsets from
    ``n_single``). ``state_rows`` holds one state row per sequence, singles first. Rows [0, n_paged) attend through the page
    tables one row at a time (``block_table`` / ``seq_lens`` per row); the portions behind them attend tile-wise over their whole
    context (``cu_q`` from row ``n_paged``, ``cu_ctx`` into ``ctx_slots``)."""

    ids: torch.Tensor
    positions: torch.Tensor          # int32 [T]
    slots: torch.Tensor              # int64 [T]: page * page size + offset, negative: not cached
    n_single: int
    n_paged: int
    block_table: torch.Tensor        # int32 [n_paged, pages]
    seq_lens: torch.Tensor           # int32 [n_paged]
    state_rows: Optional[torch.Tensor] = None   # int64 [sequences]
    cu: Optional[torch.Tensor] = None           # int32
    max_portion: int = 0
    cu_q: Optional[torch.Tensor] = None         # int32
    cu_ctx: Optional[torch.Tensor] = None       # int32
    ctx_slots: Optional[torch.Tensor] = None    # int64
    max_q: int = 0
    max_ctx: int = 0                 # upper bound of seq_lens (a host number, fixed while a graph is captured)
    num_splits: int = 1

    @property
    def rows(self) -> int:
        return self.positions.shape[0]


def _f32(t: torch.Tensor) -> int:
    return int(t.dtype == torch.float32)


def _dyt_ref(x, norm):
    return (torch.tanh(norm.alpha.float() * x) * norm.weight.float() + norm.bias.float()).to(norm.weight.dtype)


# --------------------------------------------------------------------------------------- residual stream
def embed_rows(ids, table, scale: float, step: Optional[torch.Tensor], norm, keep: bool):
    """x = table[ids] * scale (fp32; ``e`` is a copy when ``keep``), plus ``step`` when a loop begins at the first layer.
    Returns (x, e or None, norm(x))."""
    if not use_native(table):
        e = table[ids.long()].float() * scale
        x = e + step.float() if step is not None else e.clone()
        return x, (e if keep else None), _dyt_ref(x, norm)
    T, d = ids.shape[0], table.shape[1]
    dev = table.device
    x = torch.empty((T, d), dtype=torch.float32, device=dev)
    e = torch.empty_like(x) if keep else None
    h = torch.empty((T, d), dtype=table.dtype, device=dev)
    call("rlb_embed_rows", ptr(ids), int(ids.dtype == torch.int64), ptr(table), _f32(table), ptr(x), ptr(e), ptr(h), ptr(step),
         ptr(norm.alpha), ptr(norm.weight), ptr(norm.bias), T, d, table.shape[0], float(scale), ptr(_L.status_word(dev)), stream_ptr())
    return x, e, h


# --------------------------------------------------------------------------------------- products
def _rows_gemm(a, w, out, act_from=NO_ACT, x=None, e=None, step=None, norm=None):
    call("rlb_gemm_rows", ptr(a), ptr(w), ptr(out), a.shape[0], w.shape[0], w.shape[1], a.stride(0), w.stride(0), out.stride(0),
         _f32(a), _f32(out), act_from, ptr(x), x.stride(0) if x is not None else 0, ptr(e), ptr(step),
         *((ptr(norm.alpha), ptr(norm.weight), ptr(norm.bias)) if norm is not None else (None, None, None)), stream_ptr())
    return out


def in_proj(h: torch.Tensor, w: torch.Tensor, act_from: int) -> torch.Tensor:
    """h w^T with the square of relu on columns from ``act_from`` on."""
    if not use_native(h):
        p = h @ w.t()
        if act_from < p.shape[1]:
            p[:, act_from:] = torch.relu(p[:, act_from:]).square()
        return p
    return _rows_gemm(h, w, torch.empty((h.shape[0], w.shape[0]), dtype=h.dtype, device=h.device), act_from)


def out_proj_(x: torch.Tensor, a: torch.Tensor, w: torch.Tensor, e: Optional[torch.Tensor], step: Optional[torch.Tensor], norm) -> torch.Tensor:
    """x += a w^T (+ e) (+ step) in place on the fp32 residual stream; returns the dynamic-tanh norm of the result."""
    if not use_native(x):
        x += (a @ w.t()).float()
        if e is not None:
            x += e
        if step is not None:
            x += step.float()
        return _dyt_ref(x, norm)
    return _rows_gemm(a, w, torch.empty((a.shape[0], w.shape[0]), dtype=a.dtype, device=a.device), NO_ACT, x, e, step, norm)


def logits(h: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype = torch.float32) -> torch.Tensor:
    if not use_native(h):
        return (h.float() @ w.float().t()).to(out_dtype)
    return _rows_gemm(h, w, torch.empty((h.shape[0], w.shape[0]), dtype=out_dtype, device=h.device))


# --------------------------------------------------------------------------------------- latent attention
def _page_rows(table_row: torch.Tensor, n: int, block_size: int) -> torch.Tensor:
    t = torch.arange(n, device=table_row.device)
    return table_row.long()[t // block_size] * block_size + t % block_size


def latent_attention_(p: torch.Tensor, m, b: TokenBatch, cache: torch.Tensor) -> None:
    """Latent attention of all rows of ``p`` over the paged latent cache [pages, page size, width]; the rows' own latents are
    written first. ``m``: the layer's ``LatentAttentionMixer``."""
    bs = cache.shape[1]
    if not use_native(p):
        lat, kr = m.key_parts(p, b.positions)
        ok = b.slots >= 0
        rows = torch.zeros((p.shape[0], m.latent_width), dtype=p.dtype)
        rows[:, : m.rank], rows[:, m.rank : m.rank + m.rot_dim] = lat.to(p.dtype), kr.to(p.dtype)
        flat = cache.view(-1, m.latent_width)
        flat[b.slots[ok].long()] = rows[ok]
        q, H = m.queries(p, b.positions).to(p.dtype).float(), m.heads
        uk = m.kv_up[: H * m.dim].float().view(H, m.dim, m.rank)
        uv = m.kv_up[H * m.dim :].float().view(H, m.vdim, m.rank)
        for i in range(p.shape[0]):
            n = int(b.seq_lens[i])
            g = p[i, m.mix_off : m.mix_off + H * m.vdim]
            if n == 0:
                g.zero_()
                continue
            c = flat[_page_rows(b.block_table[i], n, bs)].float()
            qa = torch.cat([torch.einsum("hd,hdr->hr", q[i, :, : m.dim], uk), q[i, :, m.dim :]], dim=1)
            w = torch.softmax(qa @ c[:, : m.rank + m.rot_dim].t() * m.scale, dim=-1)
            y = torch.einsum("hr,hvr->hv", w @ c[:, : m.rank], uv).reshape(-1)
            g.copy_((y * torch.sigmoid(g.float())).to(p.dtype))
        return
    st = ptr(_L.status_word(p.device))
    call("rlb_latent_prep", ptr(p), _f32(p), p.shape[0], p.stride(0), m.q_off, m.lat_off, m.heads, m.dim, m.rot_dim, m.rank, m.latent_width, bs,
         cache.shape[0], ptr(b.positions), ptr(b.slots), ptr(m.kv_norm), ptr(m.freq), m.freq.numel(), float(m.gain), float(m.eps), ptr(cache), st,
         stream_ptr())
    call("rlb_latent_rows", ptr(p), _f32(p), b.n_paged, p.stride(0), m.q_off, m.mix_off, m.heads, m.dim, m.rot_dim, m.vdim, m.rank, m.latent_width,
         bs, cache.shape[0], ptr(cache), ptr(b.block_table), b.block_table.stride(0), ptr(b.seq_lens), ptr(m.kv_up), float(m.scale), st, stream_ptr())


# --------------------------------------------------------------------------------------- retention
def retention_(p: torch.Tensor, m, b: TokenBatch, state: torch.Tensor) -> None:
    """Retention of all rows of ``p``: every sequence's row of ``state`` [rows, heads, dim, vdim] (fp32) is advanced by its tokens. A
    piece that starts at position 0 starts from zero. ``m``: the layer's ``RetentionMixer``."""
    if not use_native(p):
        cuts = list(range(b.n_single)) + ([b.n_single + c for c in b.cu.tolist()] if b.cu is not None else [b.n_single])
        q, k, v = m.qkv(p, b.positions)
        o = torch.zeros((p.shape[0], m.heads, m.vdim))
        for j, (s, e) in enumerate(zip(cuts[:-1], cuts[1:])):
            r = int(b.state_rows[j])
            S = state[r] if int(b.positions[s]) else torch.zeros_like(state[r])
            o[s:e], state[r] = m.scan(q[s:e], k[s:e], v[s:e], S)
        p[:, m.mix_off : m.mix_off + m.heads * m.vdim] = m.finish(o, p)
        return
    st = ptr(_L.status_word(p.device))

    def run(row0, pieces, cu, rows):
        call("rlb_retention_rows", ptr(p), _f32(p), row0, pieces, p.stride(0), m.q_off, m.k_off, m.v_off, m.mix_off, m.heads, m.dim, m.vdim, ptr(cu),
             ptr(b.positions), ptr(rows), ptr(state), state.shape[0], ptr(m.decay), ptr(m.freq), m.freq.numel(), float(m.gain), m.dim ** -0.5,
             float(m.eps), st, stream_ptr())

    if b.n_single:
        run(0, b.n_single, None, b.state_rows)
    if b.cu is not None:
        run(b.n_single, b.cu.numel() - 1, b.cu, b.state_rows[b.n_single :])
