"""Operators of parallel mixer layers (``rl_b200/models/mixers.py``), and latent attention of every kind of layer, in the generation engine, over a batch of token rows that mixes
single decoded tokens and portions of prompts.

Each operator has the native sm_100a body (CUDA tensors, bf16 or fp32) and a plain PyTorch statement (CPU tensors). A layer is

    p = in_proj(h)               fused projection, squared ReLU on the MLP columns (epilogue)
    latent_* / retention_*       the mixer; writes its gated output over the gate columns of ``p``
    h = out_proj_(x, p)          x += p[gate | up] @ out_proj^T, the loop's additions and the NEXT layer's dynamic-tanh norm (epilogue)

so nothing but the two products and the mixer touches memory. fp32 models run every product in true fp32.
"""

from __future__ import annotations

from dataclasses import dataclass, field
from typing import Optional

import torch

from . import functional as F
from . import lib as _L
from .lib import F as CF
from .lib import I, L as LL, P, call, ptr, register, stream_ptr, use_native

register("rlb_embed_rows", [P, I, P, I, P, P, P, P, P, P, P, LL, I, I, CF, CF, P, P])
register("rlb_gemm_rows", [P, P, P, I, I, I, LL, LL, LL, I, I, I, P, LL, P, P, P, P, P, P])
register("rlb_gemm_layer", [P, P, P, I, I, I, LL, LL, LL, I, P, LL, P, P, P, P, P, P, P])
register("rlb_gemm_skinny_layer", [P, P, P, I, I, I, LL, LL, LL, I, P, LL, P, P, P, P, P, P, P])
register("rlb_latent_prep", [P, I, LL, LL, I, P, LL, I, I, I, I, I, I, I, I, P, P, P, P, I, I, CF, CF, P, P, I, P, P])
register("rlb_latent_gather", [P, P, P, LL, I, LL, P, P])
register("rlb_flash_latent_supported", [I, I, I, I])
register("rlb_flash_latent", [P, LL, LL, I, I, P, P, LL, I, P, P, I, I, I, I, I, I, I, P, LL, I, I, CF, I, P, P])
register("rlb_latent_decode_supported", [I, I, I, I, I, I])
register("rlb_latent_decode", [P, I, LL, I, I, P, LL, I, I, I, I, I, I, I, I, I, I, P, P, I, P, P, CF, P, P, I, P, P, P, P])
register("rlb_latent_rows", [P, I, I, LL, I, P, LL, I, I, I, I, I, I, I, I, I, I, P, P, I, P, P, CF, P, P])
register("rlb_retention_rows", [P, I, I, I, LL, I, I, I, I, I, I, I, P, P, P, P, LL, P, P, I, CF, CF, CF, P, P])
register("rlb_retention_supported", [I, I])
register("rlb_retention_step", [P, I, LL, I, I, I, I, I, I, I, P, P, P, LL, P, P, I, CF, CF, CF, P, P])
register("rlb_retention_portions", [P, LL, LL, I, I, I, I, I, I, I, I, I, I, I, P, P, P, P, P, P, LL, P, P, I, CF, CF, CF, P, P, P, P])

NO_ACT = 1 << 30
CHUNK = 128          # rows per chunk of the chunked recurrences
KEY_TILE = 64        # keys per tile of the attention of prompt portions
PAGED_PORTION = 16   # portions of at most this many tokens attend row by row over the pages (decode kernels)


def chunk_lists(lens) -> tuple:
    """(piece_chunk, chunk_row, chunk_rows) int32 of portions of ``lens`` rows that stand one after another."""
    first, row, rows, at = [0], [], [], 0
    for n in lens:
        for c in range(0, n, CHUNK):
            row.append(at + c)
            rows.append(min(CHUNK, n - c))
        at += n
        first.append(len(row))
    return tuple(torch.tensor(x, dtype=torch.int32) for x in (first, row, rows))


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
    piece_chunk: Optional[torch.Tensor] = None  # int32 [n + 1]: chunks (of at most CHUNK rows) of every portion
    chunk_row: Optional[torch.Tensor] = None    # int32: first row of every chunk, counted from n_single
    chunk_rows: Optional[torch.Tensor] = None   # int32
    cu_q: Optional[torch.Tensor] = None         # int32
    cu_ctx: Optional[torch.Tensor] = None       # int32
    ctx_slots: Optional[torch.Tensor] = None    # int64
    q_tiles: int = 0                 # 128-row query tiles of those portions
    row_off: Optional[torch.Tensor] = None      # int32 [T]: rows of the same piece before each row (None: all rows are singles)
    row_state: Optional[torch.Tensor] = None    # int64 [T]: state row of each row's sequence (None: ``state_rows``)
    whole: bool = False              # the tile-wise portions start at position 0
    chunk_ctx: dict = field(default_factory=dict)   # chunk size: (cu_ctx, ctx_slots, whole) of layers that see chunks, from the border before each portion
    window_ctx: dict = field(default_factory=dict)  # (window, kept): (cu_ctx, ctx_slots, skip) of layers that see windows, without what no row of a portion sees
    max_ctx: int = 0                 # upper bound of seq_lens (a host number, fixed while a graph is captured)

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
         ptr(norm.alpha), ptr(norm.weight), ptr(norm.bias), T, d, table.shape[0], float(scale), 0.0, ptr(_L.status_word(dev)), stream_ptr())
    return x, e, h


# --------------------------------------------------------------------------------------- products
def _aligned(*ts) -> bool:
    """bf16 matrices whose rows start on 16-byte boundaries (what TMA can fetch)."""
    return all(t.dtype == torch.bfloat16 and t.data_ptr() % 16 == 0 and t.stride(0) % 8 == 0 for t in ts)


def _product(a, w, out, act_from=NO_ACT, x=None, e=None, step=None, norm=None):
    """out = epilogue(a w^T): the tensor-core kernels for bf16 shapes that TMA can address, else the plain kernel (any size, fp32)."""
    M, (N, K) = a.shape[0], w.shape
    lay = (ptr(x), x.stride(0) if x is not None else 0, ptr(e), ptr(step),
           *((ptr(norm.alpha), ptr(norm.weight), ptr(norm.bias)) if norm is not None else (None, None, None)))
    if _aligned(a, w, out) and N % 8 == 0 and K % 8 == 0:
        name = "rlb_gemm_skinny_layer" if M <= 256 and K >= 256 else "rlb_gemm_layer"
        call(name, ptr(a), ptr(w), ptr(out), M, N, K, a.stride(0), w.stride(0), out.stride(0), act_from, *lay,
             ptr(_L.status_word(a.device)), stream_ptr())
    else:
        call("rlb_gemm_rows", ptr(a), ptr(w), ptr(out), M, N, K, a.stride(0), w.stride(0), out.stride(0), _f32(a), _f32(out), act_from, *lay,
             stream_ptr())
    return out


def in_proj(h: torch.Tensor, w: torch.Tensor, act_from: int) -> torch.Tensor:
    """h w^T with the square of relu on columns from ``act_from`` on."""
    if not use_native(h):
        p = h @ w.t()
        if act_from < p.shape[1]:
            p[:, act_from:] = torch.relu(p[:, act_from:]).square()
        return p
    return _product(h, w, torch.empty((h.shape[0], w.shape[0]), dtype=h.dtype, device=h.device), act_from)


def out_proj_(x: torch.Tensor, a: torch.Tensor, w: torch.Tensor, e: Optional[torch.Tensor], step: Optional[torch.Tensor], norm) -> torch.Tensor:
    """x += a w^T (+ e) (+ step) in place on the fp32 residual stream; returns the dynamic-tanh norm of the result."""
    if not use_native(x):
        x += (a @ w.t()).float()
        if e is not None:
            x += e
        if step is not None:
            x += step.float()
        return _dyt_ref(x, norm)
    return _product(a, w, torch.empty((a.shape[0], w.shape[0]), dtype=a.dtype, device=a.device), NO_ACT, x, e, step, norm)


def logits(h: torch.Tensor, w: torch.Tensor, out_dtype: torch.dtype = torch.float32) -> torch.Tensor:
    if not use_native(h):
        return (h.float() @ w.float().t()).to(out_dtype)
    if _aligned(h, w) and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0:
        return F.gemm(h, w, out_dtype=out_dtype)
    return _product(h, w, torch.empty((h.shape[0], w.shape[0]), dtype=out_dtype, device=h.device))


# --------------------------------------------------------------------------------------- latent attention
def _page_rows(table_row: torch.Tensor, n: int, block_size: int) -> torch.Tensor:
    t = torch.arange(n, device=table_row.device)
    return table_row.long()[t // block_size] * block_size + t % block_size


def latent_attention(p: torch.Tensor, m, b: TokenBatch, cache: torch.Tensor) -> torch.Tensor:
    """Rows [T, mix_width] of latent attention without an output gate, its queries taken from their own latent where the mixer has one
    (normed in place in ``p``)."""
    from .layer_ops import group_norm_, linear

    q = p
    if m.q_rank:
        group_norm_(p, m.q_norm, 1, m.eps)
        q = linear(p[:, : m.q_up.shape[1]], m.q_up)
    n = m.heads * m.vdim
    y = (torch.zeros if m.mix_width > n else torch.empty)((p.shape[0], m.mix_width), dtype=p.dtype, device=p.device)
    latent_attention_(p, m, b, cache, q, y)
    return y


def latent_attention_(p: torch.Tensor, m, b: TokenBatch, cache: torch.Tensor, q=None, out=None) -> None:
    """Latent attention of all rows of ``p`` over the paged latent cache [pages, page size, width]; the rows' own latents are
    written first. ``m``: the layer's ``LatentAttentionMixer``. Queries are columns of ``q`` (None: of ``p``; rotated in place), head outputs
    columns of ``out`` (None: of ``p``, over the gates)."""
    bs = cache.shape[1]
    q, out = p if q is None else q, p if out is None else out
    if not use_native(p):
        lat, kr = m.key_parts(p, b.positions)
        ok = b.slots >= 0
        rows = torch.zeros((p.shape[0], m.latent_width), dtype=p.dtype)
        rows[:, : m.rank], rows[:, m.rank : m.rank + m.rot_dim] = lat.to(p.dtype), kr.to(p.dtype)
        flat = cache.view(-1, m.latent_width)
        flat[b.slots[ok].long()] = rows[ok]
        q, H = m.queries(q, b.positions).to(p.dtype).float(), m.heads
        uk = m.kv_up[: H * m.dim].float().view(H, m.dim, m.rank)
        uv = m.kv_up[H * m.dim :].float().view(H, m.vdim, m.rank)
        for i in range(p.shape[0]):
            n = int(b.seq_lens[i])
            g = out[i, m.mix_off : m.mix_off + H * m.vdim]
            if n == 0:
                g.zero_()
                continue
            c = flat[_page_rows(b.block_table[i], n, bs)].float()
            qa = torch.cat([torch.einsum("hd,hdr->hr", q[i, :, : m.dim], uk), q[i, :, m.dim :]], dim=1)
            w = torch.softmax(qa @ c[:, : m.rank + m.rot_dim].t() * m.scale, dim=-1)
            y = torch.einsum("hr,hvr->hv", w @ c[:, : m.rank], uv).reshape(-1)
            g.copy_((y * torch.sigmoid(g.float()) if m.gate else y).to(p.dtype))
        return
    dev, T, H, W = p.device, p.shape[0], m.heads, m.latent_width
    st = ptr(_L.status_word(dev))
    decode = b.n_paged > 0 and decode_tiles(p, m, bs)
    q_lat = torch.empty((b.n_paged, H, W), dtype=p.dtype, device=dev) if decode else None
    call("rlb_latent_prep", ptr(p), _f32(p), T, p.stride(0), m.lat_off, ptr(q), q.stride(0), m.q_off, H, m.dim, m.rot_dim, m.rank, W, bs,
         cache.shape[0], ptr(b.positions), ptr(b.slots), ptr(m.kv_norm), ptr(m.freq), m.freq.numel(), int(not m.interleaved), float(m.gain), float(m.eps),
         ptr(cache), ptr(q_lat), b.n_paged if decode else 0, st, stream_ptr())
    if decode:
        splits = split_count(b.n_paged * -(-H // (32 if H > 16 else 16)), b.max_ctx)
        o_lat = torch.empty((b.n_paged, H * m.rank), dtype=p.dtype, device=dev)
        po = torch.empty(b.n_paged * H * splits * m.rank, dtype=torch.float32, device=dev) if splits > 1 else None
        pml = torch.empty(b.n_paged * H * splits * 2, dtype=torch.float32, device=dev) if splits > 1 else None
        call("rlb_latent_decode", ptr(q), b.n_paged, q.stride(0), q.shape[1], m.q_off, ptr(out), out.stride(0), m.mix_off, int(m.gate), H, m.dim, m.rot_dim, m.vdim, m.rank, W, bs,
             cache.shape[0], ptr(cache), ptr(b.block_table), b.block_table.stride(0), ptr(b.seq_lens), ptr(m.kv_up), float(m.scale), ptr(q_lat),
             ptr(o_lat), splits, ptr(po), ptr(pml), st, stream_ptr())
    elif b.n_paged:
        call("rlb_latent_rows", ptr(q), _f32(p), b.n_paged, q.stride(0), m.q_off, ptr(out), out.stride(0), m.mix_off, int(m.gate), H, m.dim, m.rot_dim, m.vdim, m.rank, W, bs,
             cache.shape[0], ptr(cache), ptr(b.block_table), b.block_table.stride(0), ptr(b.seq_lens), ptr(m.kv_up), float(m.scale), st, stream_ptr())
    if b.n_paged < T:
        n = b.ctx_slots.numel()
        lat = torch.empty((n, W), dtype=p.dtype, device=dev)
        call("rlb_latent_gather", ptr(cache), ptr(b.ctx_slots), ptr(lat), n, W, cache.shape[0] * bs, st, stream_ptr())
        kv = F.gemm(lat[:, : m.rank], m.kv_up)
        call("rlb_flash_latent", ptr(q), T, q.stride(0), q.shape[1], b.n_paged, ptr(kv), ptr(lat), n, W, ptr(b.cu_q), ptr(b.cu_ctx),
             b.cu_q.numel() - 1, H, m.dim, m.rot_dim, m.vdim, m.rank, m.q_off, ptr(out), out.stride(0), m.mix_off, int(m.gate), float(m.scale),
             b.q_tiles, st, stream_ptr())


def decode_tiles(p: torch.Tensor, m, block_size: int) -> bool:
    """Whether the tensor-core decode kernels take this layer's shape."""
    return p.dtype == torch.bfloat16 and (m.dim + m.rot_dim) % 8 == 0 and \
        bool(_L.lib().rlb_latent_decode_supported(m.dim, m.rot_dim, m.vdim, m.rank, m.latent_width, block_size))


def portion_tiles(m, dtype: torch.dtype) -> bool:
    """Whether the tensor-core prefill kernel takes this layer's shape."""
    return dtype == torch.bfloat16 and (m.dim + m.rot_dim) % 8 == 0 and (m.heads * (m.dim + m.vdim)) % 8 == 0 and \
        bool(_L.lib().rlb_flash_latent_supported(m.dim, m.rot_dim, m.vdim, m.rank))


def split_count(ctas: int, max_ctx: int, sms: int = 148) -> int:
    """Context splits of the decode attention (one CTA per SM): the count whose waves waste least, at least 256 tokens per split."""
    best, cost = 1, float("inf")
    for s in range(1, min(32, max(1, max_ctx // 256)) + 1):
        c = -(-ctas * s // sms) / s + 0.01 * s
        if c < cost - 1e-9:
            best, cost = s, c
    return best


# --------------------------------------------------------------------------------------- retention
def retention_(p: torch.Tensor, m, b: TokenBatch, state: torch.Tensor, plain: bool = False) -> None:
    """Retention of all rows of ``p``: every sequence's row of ``state`` [rows, heads, dim, vdim] (fp32) is advanced by its tokens. A
    piece that starts at position 0 starts from zero. ``m``: the layer's ``RetentionMixer``. ``plain``: the token-by-token kernel for
    every shape (it serves fp32 models and odd sizes)."""
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

    if not plain and p.dtype == torch.bfloat16 and _L.lib().rlb_retention_supported(m.dim, m.vdim):
        if b.n_single:
            call("rlb_retention_step", ptr(p), b.n_single, p.stride(0), m.q_off, m.k_off, m.v_off, m.mix_off, m.heads, m.dim, m.vdim, ptr(b.positions),
                 ptr(b.state_rows), ptr(state), state.shape[0], ptr(m.decay), ptr(m.freq), m.freq.numel(), float(m.gain), m.dim ** -0.5, float(m.eps),
                 st, stream_ptr())
        if b.cu is not None:
            n = b.chunk_row.numel()
            cs = torch.empty((p.shape[0] - b.n_single) * 2 * m.freq.numel() + 4, dtype=torch.float32, device=p.device)
            sums = torch.empty((n, m.heads, m.dim, m.vdim), dtype=torch.float32, device=p.device)
            call("rlb_retention_portions", ptr(p), p.shape[0], p.stride(0), p.shape[1], b.n_single, m.q_off, m.k_off, m.v_off, m.mix_off, m.heads, m.dim,
                 m.vdim, b.cu.numel() - 1, n, ptr(b.piece_chunk), ptr(b.chunk_row), ptr(b.chunk_rows), ptr(b.positions),
                 ptr(b.state_rows[b.n_single :]), ptr(state), state.shape[0], ptr(m.log2_decay), ptr(m.freq), m.freq.numel(), float(m.gain),
                 m.dim ** -0.5, float(m.eps), ptr(cs), ptr(sums), st, stream_ptr())
        return
    if b.n_single:
        run(0, b.n_single, None, b.state_rows)
    if b.cu is not None:
        run(b.n_single, b.cu.numel() - 1, b.cu, b.state_rows[b.n_single :])
