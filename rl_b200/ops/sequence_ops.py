"""Sequence mixers of post-norm and pre-norm layers in the generation engine: grouped-query attention over paged keys and values, and the recurrent
mixers with a short convolution (Mamba-2, gated delta rule), over a batch of token rows that mixes single decoded tokens and portions of
prompts (``mixer_ops.TokenBatch``).

Each operator takes the projected rows ``p`` of the layer's mixer module and returns the rows [T, mix_width] that its output product reads.
CUDA tensors run the native kernels: tensor-core forms for bf16 shapes they take, kernels for any size otherwise and for fp32 models;
CPU tensors run the plain PyTorch statement.
"""

from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field
from typing import Any, Optional

import torch

from . import engine_ops as E
from . import lib as _L
from .layer_ops import _pieces, group_norm_
from .lib import F as CF
from .lib import I, L as LL, P, call, ptr, register, stream_ptr, use_native
from .mixer_ops import TokenBatch, _f32, _page_rows

register("rlb_gqa_prep", [P, I, LL, LL, I, I, I, I, I, I, I, I, I, P, P, P, P, P, I, I, CF, CF, P, LL, P, I, P, P, P, P])
register("rlb_gqa_rows", [P, I, I, LL, I, I, I, I, I, I, I, P, P, P, I, P, I, I, I, P, I, CF, P, LL, P, P])
register("rlb_gqa_gather", [P, P, P, P, LL, I, I, I, I, LL, P, P])
register("rlb_flash_gqa", [P, LL, LL, I, I, P, LL, LL, I, I, I, I, P, P, I, I, I, I, I, I, I, I, I, P, P, I, CF, I, P, LL, P, P])
register("rlb_conv_rows", [P, I, LL, P, LL, LL, I, I, P, P, P, P, P, P, LL, P, P])
register("rlb_conv_state", [P, I, LL, I, I, P, I, I, P, P, P, LL, P])
register("rlb_mamba2_rows", [P, I, LL, P, LL, P, LL, I, I, I, I, I, I, I, I, P, P, P, P, LL, P, P, P, P, P])
register("rlb_delta_rows", [P, I, LL, P, LL, P, LL, I, I, I, I, I, I, I, I, I, P, P, P, P, LL, P, P, P, CF, CF, P, P])
register("rlb_rec_supported", [I, I, I])
register("rlb_conv_runs", [P, LL, P, LL, LL, I, I, P, P, P, P, P, P, LL, P, P])
register("rlb_rec_step", [P, P])
register("rlb_rec_portions", [P, P])


class _RecArgs(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("p", "u", "conv_w", "conv_bias", "A_log", "dt_bias", "D", "norm", "y", "ring", "positions", "piece_chunk",
                                          "chunk_row", "chunk_rows", "state_rows", "state", "cum", "wt", "unit", "start", "u0", "w_hi", "w_lo", "kt_hi",
                                          "kt_lo", "uu_hi", "uu_lo", "status")] + \
               [(n, C.c_longlong) for n in ("ldp", "ldu", "ldy", "num_states", "rows")] + \
               [(n, C.c_int) for n in ("delta", "heads", "groups", "dim", "vdim", "taps", "channels", "conv_off", "gate_off", "a_off", "b_off", "row0",
                                       "pieces", "chunks")] + [("unit_eps", C.c_float), ("eps", C.c_float)]


def _rows_out(p: torch.Tensor, m) -> torch.Tensor:
    n = m.heads * m.vdim
    return (torch.zeros if m.mix_width > n else torch.empty)((p.shape[0], m.mix_width), dtype=p.dtype, device=p.device)


# --------------------------------------------------------------------------------------- attention
@dataclass
class KeyValues:
    """Keys and values of one layer in one step, for the layers that read them: its projected rows (whole portions attend to those) and, by mask,
    what was gathered from its cache."""

    p: torch.Tensor
    m: Any
    gathered: dict = field(default_factory=dict)


def attention(p: torch.Tensor, m, b: TokenBatch, k_cache: torch.Tensor, v_cache: torch.Tensor, first: Optional[torch.Tensor] = None,
              kv: Optional[KeyValues] = None) -> torch.Tensor:
    """``m``: the layer's ``GroupedAttentionMixer``; caches [pages, kv_heads, page size, dim / vdim]. The rows' own keys and values are
    written first; ``p`` is left with normed and rotated queries and keys. ``first`` [T, kv_heads * vdim]: an earlier layer's values of the
    rows, of which the layer's own take over a share before they are written. A layer without keys and values of its own reads those of ``kv``, and
    the caches are that layer's. With an output gate the outputs stand over the gates in ``p``."""
    bs, H, G = k_cache.shape[2], m.heads, m.kv_heads
    own = m.kv_from is None
    if not use_native(p):
        y = _rows_out(p, m)
        q = m.queries(p, b.positions)
        if own:
            k, v = m.keys_values(p, b.positions, first)
            ok = b.slots >= 0
            page, off = (b.slots[ok] // bs).long(), (b.slots[ok] % bs).long()
            k_cache[page, :, off], v_cache[page, :, off] = k[ok].to(k_cache.dtype), v[ok].to(v_cache.dtype)
        q = q.to(p.dtype).float()
        for i in range(p.shape[0]):
            n = int(b.seq_lens[i])
            if n == 0:
                y[i] = 0
                continue
            t = torch.arange(n)
            t = t[~m.hidden(torch.tensor(n - 1), t)]
            rows = _page_rows(b.block_table[i], n, bs)[t]
            ks, vs = (c[rows // bs, :, rows % bs].float().transpose(0, 1) for c in (k_cache, v_cache))      # [kv_heads, n, dim]
            z = (q[i].view(G, H // G, m.dim) @ ks.transpose(1, 2) * m.scale).view(H, 1, -1)
            w = m.weigh(z, torch.zeros((), dtype=torch.bool)).view(G, H // G, -1)
            y[i, : H * m.vdim] = m.gated((w @ vs).reshape(1, -1), p[i : i + 1])[0].to(p.dtype)
        return y
    T, st = p.shape[0], ptr(_L.status_word(p.device))
    y = p[:, m.mix_off : m.mix_off + m.mix_width] if m.gate else _rows_out(p, m)
    call("rlb_gqa_prep", ptr(p), _f32(p), T, p.stride(0), m.q_off, m.k_off, m.v_off, H, G, m.dim, m.vdim, bs, k_cache.shape[0], ptr(b.positions),
         ptr(b.slots), ptr(m.q_norm), ptr(m.k_norm), ptr(m.freq), m.freq.numel(), int(not m.interleaved), float(m.gain), float(m.eps), ptr(first),
         first.stride(0) if first is not None else 0, ptr(m.v_share) if first is not None else None, int(own), ptr(k_cache), ptr(v_cache), st, stream_ptr())
    if b.n_paged:
        if decode_tiles(p, m, bs):
            seen = min(b.max_ctx, m.chunk) // 2 if m.chunk else min(b.max_ctx // 2, m.window + m.keep) if m.window else b.max_ctx // 2
            E.paged_decode(p[: b.n_paged, m.q_off : m.q_off + H * m.dim], k_cache, v_cache, b.block_table, b.seq_lens, H, G, m.dim, scale=m.scale,
                           num_splits=E.choose_splits(b.n_paged, G, max(seen, 1), bs), out=y[: b.n_paged], chunk=m.chunk, window=m.window, keep=m.keep,
                           offset=m.offset, gated=m.gate)
        else:
            call("rlb_gqa_rows", ptr(p), _f32(p), b.n_paged, p.stride(0), m.q_off, H, G, m.dim, m.vdim, bs, k_cache.shape[0], ptr(k_cache),
                 ptr(v_cache), ptr(b.block_table), b.block_table.stride(0), ptr(b.seq_lens), m.chunk, m.window, m.keep, ptr(m.offset), int(m.gate),
                 float(m.scale), ptr(y), y.stride(0), st, stream_ptr())
    if b.n_paged < T:
        cu_ctx, slots, whole, skip = b.cu_ctx, b.ctx_slots, b.whole, None
        if m.chunk in b.chunk_ctx:
            cu_ctx, slots, whole = b.chunk_ctx[m.chunk]
        elif not whole and (m.window, m.keep) in b.window_ctx:
            cu_ctx, slots, skip = b.window_ctx[m.window, m.keep]
        if whole:         # no cached key is visible to these portions: theirs, and their values, stand in the projected rows
            rows, row0 = T, b.n_paged
            src, k0, v0 = (p, m.k_off, m.v_off) if own else (kv.p, kv.m.k_off, kv.m.v_off)
        else:
            rows, row0, k0, v0 = slots.numel(), 0, 0, G * m.dim
            seen = (m.chunk, m.window, m.keep)
            src = kv.gathered.get(seen) if kv is not None else None
            if src is None:
                src = torch.empty((rows, G * (m.dim + m.vdim)), dtype=p.dtype, device=p.device)
                call("rlb_gqa_gather", ptr(k_cache), ptr(v_cache), ptr(slots), ptr(src), rows, G, m.dim, m.vdim, bs, k_cache.shape[0] * bs, st, stream_ptr())
                if kv is not None:
                    kv.gathered[seen] = src
        call("rlb_flash_gqa", ptr(p), T, p.stride(0), p.shape[1], b.n_paged, ptr(src), rows, src.stride(0), src.shape[1], row0, k0, v0, ptr(b.cu_q),
             ptr(cu_ctx), b.cu_q.numel() - 1, H, G, m.dim, m.vdim, m.q_off, m.chunk, m.window, m.keep, ptr(skip), ptr(m.offset), int(m.gate), float(m.scale),
             b.q_tiles, ptr(y), y.stride(0), st, stream_ptr())
    return y


def decode_tiles(p: torch.Tensor, m, block_size: int) -> bool:
    """Whether the tensor-core decode kernel takes this layer's shape."""
    return p.dtype == torch.bfloat16 and m.dim == 128 and m.vdim == 128 and m.heads // m.kv_heads <= 8 and block_size in (16, 32, 64)


def portion_tiles(m, dtype: torch.dtype) -> bool:
    """Whether the tensor-core prefill kernel takes this layer's shape."""
    return dtype == torch.bfloat16 and m.dim % 16 == 0 and m.vdim % 8 == 0 and bool(_L.lib().rlb_flash_latent_supported(m.dim, 0, m.vdim, 8))


# --------------------------------------------------------------------------------------- recurrent mixers
def recurrent(p: torch.Tensor, m, b: TokenBatch, ring: torch.Tensor, state: torch.Tensor, plain: bool = False) -> torch.Tensor:
    """Mamba-2 or delta-rule mixing of all rows: every sequence's row of ``ring`` [rows, taps, channels] (the convolution's last inputs, by
    position modulo taps) and of ``state`` [rows, heads, dim, vdim] (fp32) is advanced by its tokens; a piece that starts at position 0
    starts from zeros. ``plain``: the token-by-token kernels for every shape (they serve fp32 models and odd sizes)."""
    y = _rows_out(p, m)
    if not use_native(p):
        return _recurrent_ref(p, m, b, ring, state, y)
    if not plain and rec_tiles(p, m):
        _recurrent_tiles(p, m, b, ring, state, y)
        if m.kind == "mamba2":
            group_norm_(y, m.norm, m.norm_groups, m.eps)
        return y
    st, T = ptr(_L.status_word(p.device)), p.shape[0]
    x = p[:, m.conv_off : m.conv_off + m.channels]
    u = torch.empty((T, -(-m.channels // 8) * 8), dtype=p.dtype, device=p.device)
    call("rlb_conv_rows", ptr(x), _f32(p), p.stride(0), ptr(u), u.stride(0), T, m.channels, m.taps, ptr(m.conv), ptr(m.conv_bias), ptr(ring),
         ptr(b.positions), ptr(b.row_off), ptr(b.row_state if b.row_state is not None else b.state_rows), ring.shape[0], st, stream_ptr())
    for row0, pieces, cu, rows in ((0, b.n_single, None, b.state_rows),
                                   (b.n_single, b.cu.numel() - 1 if b.cu is not None else 0, b.cu, b.state_rows[b.n_single :])):
        if not pieces:
            continue
        if m.taps > 1:
            call("rlb_conv_state", ptr(x), _f32(p), p.stride(0), row0, pieces, ptr(cu), m.channels, m.taps, ptr(ring), ptr(b.positions), ptr(rows),
                 ring.shape[0], stream_ptr())
        if m.kind == "mamba2":
            call("rlb_mamba2_rows", ptr(u), _f32(p), u.stride(0), ptr(p), p.stride(0), ptr(y), y.stride(0), m.z_off, m.dt_off, m.heads, m.groups, m.dim,
                 m.vdim, row0, pieces, ptr(cu), ptr(b.positions), ptr(rows), ptr(state), state.shape[0], ptr(m.A_log), ptr(m.dt_bias), ptr(m.D), st,
                 stream_ptr())
        else:
            call("rlb_delta_rows", ptr(u), _f32(p), u.stride(0), ptr(p), p.stride(0), ptr(y), y.stride(0), m.g_off, m.b_off, m.a_off, m.heads,
                 m.kv_heads, m.dim, m.vdim, row0, pieces, ptr(cu), ptr(b.positions), ptr(rows), ptr(state), state.shape[0], ptr(m.A_log),
                 ptr(m.dt_bias), ptr(m.norm), float(m.unit_eps), float(m.eps), st, stream_ptr())
    if m.kind == "mamba2":
        group_norm_(y, m.norm, m.norm_groups, m.eps)
    return y


def rec_tiles(p: torch.Tensor, m) -> bool:
    """Whether the tensor-core and single-step kernels take this layer's shape."""
    return p.dtype == torch.bfloat16 and m.conv_off % 8 == 0 and p.stride(0) % 8 == 0 and \
        bool(_L.lib().rlb_rec_supported(int(m.kind == "delta"), m.dim, m.vdim))


def _recurrent_tiles(p, m, b, ring, state, y) -> None:
    dev, T, delta = p.device, p.shape[0], m.kind == "delta"
    H, G = m.heads, m.kv_heads if delta else m.groups
    st = ptr(_L.status_word(dev))
    a = _RecArgs()
    a.p, a.y, a.ldp, a.ldy, a.rows, a.status = ptr(p), ptr(y), p.stride(0), y.stride(0), T, st
    a.conv_w, a.conv_bias, a.A_log, a.dt_bias, a.norm = ptr(m.conv), ptr(m.conv_bias), ptr(m.A_log), ptr(m.dt_bias), ptr(m.norm) if delta else None
    a.D = None if delta else ptr(m.D)
    a.ring, a.state, a.num_states, a.positions = ptr(ring), ptr(state), state.shape[0], ptr(b.positions)
    a.delta, a.heads, a.groups, a.dim, a.vdim, a.taps, a.channels, a.conv_off = int(delta), H, G, m.dim, m.vdim, m.taps, m.channels, m.conv_off
    a.gate_off, a.a_off, a.b_off = (m.g_off, m.a_off, m.b_off) if delta else (m.z_off, m.dt_off, -1)
    a.unit_eps, a.eps = float(m.unit_eps) if delta else 0.0, float(m.eps)
    if b.n_single:
        a.pieces, a.state_rows = b.n_single, ptr(b.state_rows)
        call("rlb_rec_step", C.byref(a), stream_ptr())
    if b.cu is None:
        return
    n0, n, pieces = b.n_single, b.chunk_row.numel(), b.cu.numel() - 1
    R, x = T - n0, p[n0:, m.conv_off : m.conv_off + m.channels]
    u = torch.empty((T, -(-m.channels // 8) * 8), dtype=p.dtype, device=dev)
    uv, rows = u[n0:], b.state_rows[n0:]
    if 2 <= m.taps <= 4 and m.channels % 8 == 0:
        call("rlb_conv_runs", ptr(x), p.stride(0), ptr(uv), u.stride(0), R, m.channels, m.taps, ptr(m.conv), ptr(m.conv_bias), ptr(ring),
             ptr(b.positions[n0:]), ptr(b.row_off[n0:]), ptr(b.row_state[n0:]), ring.shape[0], st, stream_ptr())
    else:
        call("rlb_conv_rows", ptr(x), 0, p.stride(0), ptr(uv), u.stride(0), R, m.channels, m.taps, ptr(m.conv), ptr(m.conv_bias), ptr(ring),
             ptr(b.positions[n0:]), ptr(b.row_off[n0:]), ptr(b.row_state[n0:]), ring.shape[0], st, stream_ptr())
    if m.taps > 1:
        call("rlb_conv_state", ptr(p[:, m.conv_off :]), 0, p.stride(0), n0, pieces, ptr(b.cu), m.channels, m.taps, ptr(ring), ptr(b.positions), ptr(rows),
             ring.shape[0], stream_ptr())
    f32 = lambda *s: torch.empty(s, dtype=torch.float32, device=dev)   # noqa: E731
    cw, start = f32(2, H, R), f32(n, H, m.dim, m.vdim)
    a.cum, a.wt, a.start = ptr(cw[0]), ptr(cw[1]), ptr(start)
    if delta:
        unit, u0 = f32(2, G, R), f32(n * H, 128, m.vdim)
        tiles, writes = torch.empty((4, n * H * 128, 128), dtype=p.dtype, device=dev), torch.empty((2, R, H * m.vdim), dtype=p.dtype, device=dev)
        a.unit, a.u0 = ptr(unit), ptr(u0)
        a.w_hi, a.w_lo, a.kt_hi, a.kt_lo = (ptr(t) for t in tiles)
        a.uu_hi, a.uu_lo = ptr(writes[0]), ptr(writes[1])
    a.u, a.ldu, a.row0, a.pieces, a.chunks, a.state_rows = ptr(u), u.stride(0), n0, pieces, n, ptr(rows)
    a.piece_chunk, a.chunk_row, a.chunk_rows = ptr(b.piece_chunk), ptr(b.chunk_row), ptr(b.chunk_rows)
    call("rlb_rec_portions", C.byref(a), stream_ptr())


def _recurrent_ref(p, m, b, ring, state, y):
    n = m.taps - 1
    for j, (s, e) in enumerate(_pieces(b)):
        r, pos = int(b.state_rows[j]), int(b.positions[s])
        before = torch.stack([ring[r, t % m.taps] if t >= 0 else torch.zeros_like(ring[r, 0]) for t in range(pos - n, pos)]) if n else p.new_zeros(0, m.channels)
        x = p[s:e, m.conv_off : m.conv_off + m.channels]
        u = m.convolve(x, before)
        S = state[r] if pos else torch.zeros_like(state[r])
        o, S = m.scan(u, p[s:e], S)
        y[s:e, : m.heads * m.vdim] = m.finish(o, p[s:e]).reshape(e - s, -1)
        state[r] = S
        for t in range(max(s, e - n), e):
            ring[r, (pos + t - s) % m.taps] = x[t - s]
    return y
