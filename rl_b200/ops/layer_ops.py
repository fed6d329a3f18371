"""Row operators of post-norm and pre-norm layers (``rl_b200/models/post_norm.py``, ``pre_norm.py``) in the generation engine: products with
what follows them, the join with the residual stream, the blend with the token before, the feed-forwards and the token input.

Each operator has the native sm_100a body (CUDA tensors, bf16 or fp32) and a plain PyTorch statement (CPU tensors). ``x`` is the fp32
residual stream, updated in place; ``h`` what the next sublayer reads (x in the model's type). fp32 models run every product in true fp32.
"""

from __future__ import annotations

import ctypes as C
from dataclasses import dataclass
from typing import Optional

import torch
import torch.nn.functional as TF

from . import functional as F
from . import lib as _L
from .lib import F as CF
from .lib import I, L as LL, P, call, ptr, register, stream_ptr, use_native
from .mixer_ops import TokenBatch, _aligned, _f32

register("rlb_linear_rows", [P, P])
register("rlb_linear_tiled", [P, P])
register("rlb_linear_skinny", [P, P])
register("rlb_linear_grouped", [P, P])
register("rlb_add_normed", [P, P])
register("rlb_shift_rows", [P, P, P])
register("rlb_blend_rows", [P, P, P, P, I, LL, I, P, P])
register("rlb_commit_states", [P, P, LL, P, P, P, I, LL, P, P])
register("rlb_poly_norm_rows", [P, LL, I, P, LL, I, CF, P])
register("rlb_group_norm_rows", [P, LL, I, P, LL, I, I, CF, P])
register("rlb_cap_rows", [P, LL, CF, CF, P])
register("rlb_moe_choose", [P, LL, I, I, P, I, I, I, I, CF, I, P, P, P, P, P, P, P])
register("rlb_moe_place", [P, P, LL, I, P, I, I, P, P, P, P, LL, P, I, P, P, P, P])

NONE, GLU, GELU_MUL, CAP, SILU = range(5)      # what follows a product (RlbLinearAct)


class _Linear(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("a", "w", "out", "bias", "table", "ids", "tile_expert", "a_rows", "status", "row_scale")] + \
               [(n, C.c_longlong) for n in ("lda", "ldw", "ldo", "ld_table")] + \
               [(n, C.c_int) for n in ("M", "N", "K", "in_f32", "out_f32", "act", "table_off", "table_cols", "vocab", "ids64", "experts", "num_a_rows")] + \
               [(n, C.c_float) for n in ("limit", "scale", "cap")]


def _desc(a, w, out, act=NONE, limit=0.0, bias=None) -> _Linear:
    d = _Linear()
    d.a, d.w, d.out, d.bias, d.status = ptr(a), ptr(w), ptr(out), ptr(bias), ptr(_L.status_word(a.device))
    d.M, (d.N, d.K) = a.shape[0], w.shape[-2:]
    d.lda, d.ldw, d.ldo = a.stride(0), w.stride(-2), out.stride(0)
    d.in_f32, d.out_f32, d.act, d.limit = _f32(a), _f32(out), act, limit
    return d


def _run(d: _Linear, fast: bool) -> None:
    name = "rlb_linear_rows"
    if fast and d.N % 8 == 0 and d.K % 8 == 0:
        if d.M <= 256 and d.K >= 256:
            name = "rlb_linear_skinny"
        elif not d.out_f32:
            name = "rlb_linear_tiled"
    call(name, C.byref(d), stream_ptr())


def clamped_glu_ref(p: torch.Tensor, limit: float) -> torch.Tensor:
    g, u = p[:, 0::2].float().clamp(max=limit), p[:, 1::2].float().clamp(-limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1)).to(p.dtype)


def silu_glu_ref(p: torch.Tensor) -> torch.Tensor:
    return (TF.silu(p[:, 0::2].float()) * p[:, 1::2].float()).to(p.dtype)


def gated_ref(p: torch.Tensor, limit: Optional[float]) -> torch.Tensor:
    """Gated unit over neighbouring columns: clamped to ``limit``, or silu without limits (None)."""
    return silu_glu_ref(p) if limit is None else clamped_glu_ref(p, limit)


def gated_linear(a: torch.Tensor, w: torch.Tensor, limit: Optional[float]) -> torch.Tensor:
    """``gated_ref`` of a w^T, in the product's epilogue."""
    if not use_native(a):
        return gated_ref(a @ w.t(), limit)
    out = torch.empty((a.shape[0], w.shape[0] // 2), dtype=a.dtype, device=a.device)
    _run(_desc(a, w, out, SILU if limit is None else GLU, limit or 0.0), _aligned(a, w, out))
    return out


def linear(a: torch.Tensor, w: torch.Tensor, bias: Optional[torch.Tensor] = None, glu: Optional[float] = None) -> torch.Tensor:
    """a w^T (+ bias); ``glu``: the limit of a clamped gated unit over neighbouring columns, half as wide."""
    if not use_native(a):
        p = a @ w.t() if bias is None else a @ w.t() + bias
        return p if glu is None else clamped_glu_ref(p, glu)
    out = torch.empty((a.shape[0], w.shape[0] // (1 if glu is None else 2)), dtype=a.dtype, device=a.device)
    _run(_desc(a, w, out, NONE if glu is None else GLU, glu or 0.0, bias), _aligned(a, w, out))
    return out


# --------------------------------------------------------------------------------------- residual stream
def embed(ids: torch.Tensor, table: torch.Tensor, scale: float, norm: Optional[torch.Tensor] = None, eps: float = 0.0):
    """(x, h): the tokens' rows in fp32, and in the model's type as they are or rms(x) * norm."""
    if not use_native(table):
        x = table[ids.long()].float() * scale
        return x, (x if norm is None else _rms(x, eps) * norm.float()).to(table.dtype)
    T, d = ids.shape[0], table.shape[1]
    x = torch.empty((T, d), dtype=torch.float32, device=table.device)
    h = torch.empty((T, d), dtype=table.dtype, device=table.device)
    call("rlb_embed_rows", ptr(ids), int(ids.dtype == torch.int64), ptr(table), _f32(table), ptr(x), None, ptr(h), None, None, ptr(norm), None, T, d,
         table.shape[0], float(scale), float(eps), ptr(_L.status_word(table.device)), stream_ptr())
    return x, h


def _rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps)


class _Join(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("x", "y", "copy_row", "weight", "counts", "w", "ls", "next_w", "also", "own", "also_f", "own_f", "h", "x_out", "rstd")] + \
               [(n, C.c_longlong) for n in ("ldy", "ld_also", "ld_own", "rows")] + [(n, C.c_int) for n in ("f32", "k", "y_rows", "experts", "d")] + \
               [(n, C.c_float) for n in ("mult", "eps")]


class _Shift(C.Structure):
    _fields_ = [(n, C.c_void_p) for n in ("s", "positions", "row_off", "row_state", "state", "next", "ids", "table", "pairs", "token", "token_next", "status")] + \
               [(n, C.c_longlong) for n in ("num_states", "ld_state", "mul_prev", "mul_cur")] + [(n, C.c_int) for n in ("n_single", "vocab", "buckets")] + \
               [("scale", C.c_float)]


class Carry:
    """What sequences carry from step to step beside their cache pages, a row per sequence: the normed stream of their last token at every place
    where the next token blends it in (``state`` [rows, places, d], fp32), and the token itself. Portions leave theirs in second buffers until the
    step is through (``commit``): another CTA may still have to read the old one."""

    def __init__(self, rows: int, places: int, d: int, tokens: bool, device):
        self.state = torch.zeros((rows, places, d), dtype=torch.float32, device=device) if places else None
        self.next = torch.zeros_like(self.state) if places else None
        self.token = torch.zeros(rows, dtype=torch.int32, device=device) if tokens else None
        self.token_next = torch.zeros_like(self.token) if tokens else None
        self.rows = rows

    def commit(self, b: TokenBatch) -> None:
        """Takes over what the portions of ``b`` left."""
        rows = b.state_rows[b.n_single :]
        if not rows.numel() or not rows.is_cuda:
            return
        call("rlb_commit_states", ptr(self.state), ptr(self.next), self.state[0].numel() if self.state is not None else 0, ptr(self.token), ptr(self.token_next),
             ptr(rows), rows.numel(), self.rows, ptr(_L.status_word(rows.device)), stream_ptr())


@dataclass
class Shift:
    """Blend of a normed stream with that of the token before: h + (h' - h) * s, at one of the ``places`` of ``carry`` (s None: no blend)."""

    s: Optional[torch.Tensor]
    place: int
    carry: Carry
    b: TokenBatch


FUSED_SHIFT_ROWS = 148 * 4      # fewer rows are blended by the kernel that joins or embeds them, more in a pass of their own


def _blend_after(T: int, d: int, t: Optional[Shift]) -> bool:
    return t is not None and t.s is not None and T >= FUSED_SHIFT_ROWS and d % 4 == 0 and d <= 4096


def _pieces(b: TokenBatch) -> list:
    cuts = list(range(b.n_single)) + ([b.n_single + c for c in b.cu.tolist()] if b.cu is not None else [b.n_single])
    return list(zip(cuts[:-1], cuts[1:]))


def _shift_ref(h: torch.Tensor, t: Shift) -> torch.Tensor:
    """``h`` fp32."""
    if t.s is None:
        return h
    before, state = torch.cat([h[:1], h[:-1]]), t.carry.state[:, t.place]
    for j, (s, e) in enumerate(_pieces(t.b)):
        r = int(t.b.state_rows[j])
        before[s] = state[r] if int(t.b.positions[s]) else 0.0
        state[r] = h[e - 1]
    return h + (before - h) * t.s.float()


def _shift_desc(t: Shift) -> _Shift:
    b, c, q = t.b, t.carry, _Shift()
    q.s, q.positions, q.row_off, q.n_single = ptr(t.s), ptr(b.positions), ptr(b.row_off), b.n_single
    q.row_state = ptr(b.row_state if b.row_state is not None else b.state_rows)
    q.num_states, q.status = c.rows, ptr(_L.status_word(b.positions.device))
    if t.s is not None:
        q.state, q.next, q.ld_state = ptr(c.state[:, t.place]), ptr(c.next[:, t.place]), c.state.stride(0)
    return q


def start(b: TokenBatch, table: torch.Tensor, scale: float, norm: torch.Tensor, eps: float, pairs: Optional[torch.Tensor], bigram: Optional[dict], t: Shift):
    """(x, h): the tokens' rows of ``table`` times ``scale`` plus, with ``pairs``, the rows of (token before, token) in the pair table, and rms(x) *
    norm blended by ``t``. Sequences' last tokens are kept in ``t.carry``."""
    c, T = t.carry, b.rows
    if not use_native(table):
        x = table[b.ids.long()].float() * scale
        if pairs is not None:
            rows = torch.empty(T, dtype=torch.int64)
            for j, (s, e) in enumerate(_pieces(b)):
                r, ids = int(b.state_rows[j]), b.ids[s:e].long()
                before = torch.cat([c.token[r : r + 1].long(), ids[:-1]])
                rows[s:e] = (before * bigram["mul_prev"] + ids * bigram["mul_cur"]) % bigram["buckets"]
                if int(b.positions[s]) == 0:
                    rows[s] = bigram["buckets"]
                c.token[r] = int(ids[-1])
            x = x + pairs[rows].float()
        return x, _shift_ref(_rms(x, eps) * norm.float(), t).to(table.dtype)
    d = table.shape[1]
    x = torch.empty((T, d), dtype=torch.float32, device=table.device)
    h = torch.empty((T, d), dtype=table.dtype, device=table.device)
    j, q = _Join(), _shift_desc(t)
    j.x_out, j.h, j.next_w, j.rows, j.d, j.f32, j.eps = ptr(x), ptr(h), ptr(norm), T, d, _f32(table), eps
    ids = b.ids if b.ids.dtype == torch.int32 else b.ids.int()
    q.ids, q.table, q.vocab, q.scale = ptr(ids), ptr(table), table.shape[0], float(scale)
    if pairs is not None:
        q.pairs, q.buckets, q.mul_prev, q.mul_cur = ptr(pairs), bigram["buckets"], bigram["mul_prev"], bigram["mul_cur"]
        q.token, q.token_next = ptr(c.token), ptr(c.token_next)
    after = torch.empty(T, dtype=torch.float32, device=x.device) if _blend_after(T, d, t) else None
    j.rstd = ptr(after)
    call("rlb_shift_rows", C.byref(j), C.byref(q), stream_ptr())
    if after is not None:
        call("rlb_blend_rows", ptr(x), ptr(after), ptr(norm), ptr(h), _f32(h), T, d, C.byref(q), stream_ptr())
    return x, h


def join(x: torch.Tensor, y: torch.Tensor, w: Optional[torch.Tensor], mult: float, eps: float, next_norm: Optional[torch.Tensor] = None,
         experts: Optional[tuple] = None, also: Optional[torch.Tensor] = None, also_f: Optional[torch.Tensor] = None, own: Optional[torch.Tensor] = None,
         own_f: Optional[torch.Tensor] = None, ls: Optional[torch.Tensor] = None, shift: Optional[Shift] = None):
    """(x, h) with x + mult * rms(y) * w * ls (w None: mult * y; ls None: ones) and h: x in the model's type, or rms(x) * next_norm, blended by
    ``shift``. x is updated in place, or with ``shift`` moves to a new buffer. ``experts`` = (row of every copy, weight of every copy or None, the
    experts' counts to reset): y holds expert rows, a token's value is the (weighted) sum of its copies' rows. ``also`` / ``own``: rows added to y
    first, times ``also_f`` (None: 1) / ``own_f`` [T]."""
    if not use_native(x):
        y = y.float()
        if also is not None:
            y = y + also.float() * (1.0 if also_f is None else also_f[:, None])
        if own is not None:
            y = y + own.float() * own_f[:, None]
        z = mult * (y if w is None else _rms(y, eps) * w.float())
        x += z if ls is None else z * ls.float()
        h = x if next_norm is None else _rms(x, eps) * next_norm.float()
        return x, (h if shift is None else _shift_ref(h, shift)).to((next_norm if w is None else w).dtype)
    T, d = x.shape
    h = torch.empty((T, d), dtype=y.dtype, device=x.device)
    after = torch.empty(T, dtype=torch.float32, device=x.device) if _blend_after(T, d, shift) else None
    out = x if shift is None or after is not None else torch.empty_like(x)
    rows, wt, counts = experts if experts is not None else (None, None, None)
    j = _Join()
    j.x, j.y, j.copy_row, j.weight, j.counts, j.w, j.ls, j.next_w = ptr(x), ptr(y), ptr(rows), ptr(wt), ptr(counts), ptr(w), ptr(ls), ptr(next_norm)
    j.also, j.also_f, j.own, j.own_f, j.h, j.x_out = ptr(also), ptr(also_f), ptr(own), ptr(own_f), ptr(h), ptr(out)
    j.ldy, j.ld_also, j.ld_own, j.rows, j.d = y.stride(0), also.stride(0) if also is not None else 0, own.stride(0) if own is not None else 0, T, d
    j.f32, j.k, j.y_rows, j.experts = _f32(y), rows.shape[1] if rows is not None else 0, y.shape[0], counts.numel() if counts is not None else 0
    j.mult, j.eps, j.rstd = mult, eps, ptr(after)
    if shift is None:
        call("rlb_add_normed", C.byref(j), stream_ptr())
    elif after is not None:
        call("rlb_add_normed", C.byref(j), stream_ptr())
        q = _shift_desc(shift)
        call("rlb_blend_rows", ptr(out), ptr(after), ptr(next_norm), ptr(h), _f32(h), T, d, C.byref(q), stream_ptr())
    else:
        q = _shift_desc(shift)
        call("rlb_shift_rows", C.byref(j), C.byref(q), stream_ptr())
    return out, h


def add_normed_(x: torch.Tensor, y: torch.Tensor, w: Optional[torch.Tensor], mult: float, eps: float, next_norm: Optional[torch.Tensor] = None,
                experts: Optional[tuple] = None, also: Optional[torch.Tensor] = None) -> torch.Tensor:
    """``join`` in place; returns h."""
    return join(x, y, w, mult, eps, next_norm, experts, also)[1]


def group_norm_(y: torch.Tensor, w: torch.Tensor, groups: int, eps: float) -> None:
    """The leading w.numel() columns of ``y`` in ``groups`` equal parts, each over its root mean square, times w; in place."""
    n = w.numel()
    if not use_native(y):
        y[:, :n] = (_rms(y[:, :n].float().view(y.shape[0], groups, -1), eps).reshape(-1, n) * w.float()).to(y.dtype)
        return
    call("rlb_group_norm_rows", ptr(y), y.stride(0), _f32(y), ptr(w), y.shape[0], groups, n // groups, float(eps), stream_ptr())


# --------------------------------------------------------------------------------------- feed-forwards
def feed_forward_(x: torch.Tensor, h: torch.Tensor, ff, norm: Optional[torch.Tensor], mult: float, eps: float, next_norm=None) -> torch.Tensor:
    """x += mult * rms(ff(h)) * norm (norm None: mult * ff(h)). ``ff``: the layer's feed-forward module."""
    return feed_forward(x, h, ff, norm, mult, eps, next_norm)[1]


def feed_forward(x: torch.Tensor, h: torch.Tensor, ff, norm: Optional[torch.Tensor], mult: float, eps: float, next_norm=None, ls=None, shift: Optional[Shift] = None):
    """``join`` of the feed-forward's output with the stream."""
    if hasattr(ff, "router"):
        shared = unit(h, ff.shared) if ff.shared is not None else None
        y, experts, own_f, gate = gated_experts(h, ff)
        return join(x, y, norm, mult, eps, next_norm, experts, shared, gate, h if own_f is not None else None, own_f, ls, shift)
    return join(x, poly_unit(h, ff) if hasattr(ff, "coef") else unit(h, ff), norm, mult, eps, next_norm, ls=ls, shift=shift)


def unit(h: torch.Tensor, m) -> torch.Tensor:
    return linear(gated_linear(h, m.gate_up, m.limit), m.down)


def poly_unit(h: torch.Tensor, m) -> torch.Tensor:
    """``m``: a ``PolyUnit``. (The padding columns of the first product are zeros, and so are the weights that read them.)"""
    return linear(poly_norm_(linear(h, m.up), m.coef, m.ff, m.eps), m.down)


def poly_norm_(z: torch.Tensor, coef: torch.Tensor, n: int, eps: float) -> torch.Tensor:
    """The leading n columns of ``z`` become c0 N(z) + c1 N(z^2) + c2 N(z^3) + c3, N dividing a row by its root mean square; in place."""
    if not use_native(z):
        v, c = z[:, :n].float(), coef.float()
        z[:, :n] = (c[0] * _rms(v, eps) + c[1] * _rms(v ** 2, eps) + c[2] * _rms(v ** 3, eps) + c[3]).to(z.dtype)
        return z
    call("rlb_poly_norm_rows", ptr(z), z.stride(0), _f32(z), ptr(coef), z.shape[0], n, float(eps), stream_ptr())
    return z


def gated_experts(h: torch.Tensor, m):
    """Routed part of ``m`` (``GatedExperts``): (y, experts, weight of the token's own row [T] or None, factor of the shared unit [T] or None).
    Native path: y are expert rows, experts = (row of every copy, weights or None, counts); otherwise y are summed outputs and experts None.
    Weights on the experts' inputs are factors of the first product's rows."""
    T, d = h.shape
    E, k, n = m.experts, m.top, m.outputs
    if not use_native(h):
        z = h.float() @ m.router.float().t()
        w, idx = m.choose(z[:, :n])
        y = torch.zeros((T, d), dtype=torch.float32)
        for e in range(E):
            tok, slot = (idx == e).nonzero(as_tuple=True)
            if tok.numel():
                p, wt = h[tok] @ m.gate_up[e].t(), w[tok, slot, None]
                a = gated_ref((p.float() * wt).to(p.dtype) if m.weigh_input else p, m.limit)
                y.index_add_(0, tok, (a @ m.down[e].t()).float() * (1.0 if m.weigh_input else wt))
        return y, None, (w * (idx >= E)).sum(-1) if m.identity else None, torch.sigmoid(z[:, n]) if m.shared_gate else None
    dev = h.device
    st = ptr(_L.status_word(dev))
    z = router_logits(h, m.router)
    wt = torch.empty((T, k), dtype=torch.float32, device=dev)
    idx, rank, copy_row = torch.empty((3, T, k), dtype=torch.int32, device=dev)
    own_f = torch.empty(T, dtype=torch.float32, device=dev) if m.identity else None
    gate = torch.empty(T, dtype=torch.float32, device=dev) if m.shared_gate else None
    counts = _expert_counts(m, dev)
    call("rlb_moe_choose", ptr(z), z.stride(0), T, n, ptr(m.correction), m.groups, m.keep, k, int(m.softmax), m.scale, E, ptr(wt), ptr(idx), ptr(rank), ptr(counts),
         ptr(own_f), ptr(gate), stream_ptr())
    mpad = -(-(T * k + E * 127) // 128) * 128
    tiles = torch.empty(mpad // 128, dtype=torch.int32, device=dev)
    fast = _aligned(h, m.gate_up[0], m.down[0]) and m.gate_up.shape[1] % 8 == 0 and d % 8 == 0
    xp = torch.empty((mpad, d), dtype=h.dtype, device=dev) if fast else h
    src = None if fast else torch.full((mpad,), -1, dtype=torch.int32, device=dev)
    factor = torch.empty(mpad, dtype=torch.float32, device=dev) if m.weigh_input else None
    call("rlb_moe_place", ptr(idx), ptr(rank), T * k, k, ptr(counts), E, mpad, ptr(copy_row), ptr(tiles), ptr(src), ptr(h),
         h.stride(0) * h.element_size() if fast else 0, ptr(xp) if fast else None, d * h.element_size() if fast else 0, ptr(wt) if m.weigh_input else None,
         ptr(factor), st, stream_ptr())
    a = torch.empty((mpad, m.down.shape[2]), dtype=h.dtype, device=dev)
    y = torch.empty((mpad, d), dtype=h.dtype, device=dev)
    for first, inp, w, out in ((True, xp, m.gate_up, a), (False, a, m.down, y)):
        q = _desc(inp, w, out, NONE if not first else SILU if m.limit is None else GLU, m.limit or 0.0)
        q.M, q.experts, q.tile_expert = mpad, E, ptr(tiles)
        if first:
            q.row_scale = ptr(factor)
        if first and not fast:
            q.a_rows, q.num_a_rows = ptr(src), T
        call("rlb_linear_grouped" if fast else "rlb_linear_rows", C.byref(q), stream_ptr())
    return y, (copy_row, None if m.weigh_input else wt, counts), own_f, gate


def router_logits(h: torch.Tensor, router: torch.Tensor) -> torch.Tensor:
    if _aligned(h, router) and router.shape[0] % 8 == 0 and router.shape[1] % 8 == 0:
        return F.gemm(h, router, out_dtype=torch.float32)
    z = torch.empty((h.shape[0], router.shape[0]), dtype=torch.float32, device=h.device)
    _run(_desc(h, router, z), False)
    return z


_COUNTS: dict = {}


def _expert_counts(m, dev) -> torch.Tensor:
    """Zeros that the router counts in and the join resets: one buffer per device serves all layers of a stream's step."""
    c = _COUNTS.get((dev, m.experts))
    if c is None:
        c = _COUNTS[(dev, m.experts)] = torch.zeros(m.experts, dtype=torch.int32, device=dev)
    return c


# --------------------------------------------------------------------------------------- token input, logits
def token_side_(x: torch.Tensor, h: torch.Tensor, ids: torch.Tensor, layer, table: torch.Tensor, mult: float, eps: float, next_norm=None) -> torch.Tensor:
    """x += mult * rms(proj(gelu(gate h) * e)) * norm with e the tokens' rows of the layer's columns of ``table``."""
    n, off = layer.side_dim, layer.layer_idx * layer.side_dim
    if not use_native(h):
        e = table[ids.long()][:, off : off + n].float()
        g = TF.pad(TF.gelu((h @ layer.side_gate.t()).float(), approximate="tanh")[:, :n] * e, (0, layer.side_gate.shape[0] - n)).to(h.dtype)
    else:
        g = torch.empty((h.shape[0], layer.side_gate.shape[0]), dtype=h.dtype, device=h.device)
        d = _desc(h, layer.side_gate, g, GELU_MUL)
        d.table, d.ld_table, d.table_off, d.table_cols, d.vocab = ptr(table), table.stride(0), off, n, table.shape[0]
        d.ids, d.ids64 = ptr(ids), int(ids.dtype == torch.int64)
        _run(d, _aligned(h, layer.side_gate, g))
    return add_normed_(x, linear(g, layer.side_proj), layer.side_norm, mult, eps, next_norm)


def capped_logits(h: torch.Tensor, w: torch.Tensor, scale: float, cap: float, out_dtype: torch.dtype = torch.float32) -> torch.Tensor:
    """(h w^T) * scale, soft-capped where cap > 0."""
    if not use_native(h):
        z = (h.float() @ w.float().t()) * scale
        return (cap * torch.tanh(z / cap) if cap else z).to(out_dtype)
    z = torch.empty((h.shape[0], w.shape[0]), dtype=torch.float32, device=h.device)
    ok = _aligned(h, w) and w.shape[0] % 8 == 0 and w.shape[1] % 8 == 0
    if ok and (h.shape[0] > 256 or h.shape[1] < 256):
        F.gemm(h, w, out=z)
        call("rlb_cap_rows", ptr(z), z.numel(), float(scale), float(cap), stream_ptr())
    elif z.numel():
        d = _desc(h, w, z, CAP)
        d.scale, d.cap = float(scale), float(cap)
        _run(d, ok)
    return z.to(out_dtype)
