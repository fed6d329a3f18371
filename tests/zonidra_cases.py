"""Small Zonidra models with random weights for the tests: configuration, tensors, checkpoint folder, oracle logits."""

from __future__ import annotations

import gadarax_cases as G
import torch
import zonidra_oracle as O

engine, tokens, gap, run_cut, run_schedule, mixed_schedule, live_pages, save, load = (
    G.engine, G.tokens, G.gap, G.run_cut, G.run_schedule, G.mixed_schedule, G.live_pages, G.save, G.load)

LONG = {"factor": 3.0, "low": 1.0, "high": 4.0, "original": 60}


def attention(heads=4, kv_heads=2, dim=24, vdim=16, rot_dims=16, base=10000.0, scaling=LONG, scale=0.3, size=24, keep=3, source=None):
    rot = {"dims": rot_dims, "base": base}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": dict(rot, scaling=scaling) if scaling else rot}
    if size:
        m["mask"] = {"size": size, "keep_first": keep}
    if source is not None:
        m["kv_from"] = source
    return {"type": "attention", "mixer": m}


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def moe(experts=7, identity=2, top=3, ff=20, shared=28, scale=1.7):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "identity": identity, "top": top, "scale": scale}}
    return dict(m, shared={"ff": shared}) if shared else m


def config(layers, width=56, vocab=88, scale=1.9, eps=1e-4, bigram=(101, 37, 5)):
    """``layers``: (mixer entry, feed-forward or None) pairs."""
    emb = {"scale": scale}
    if bigram:
        emb["bigram"] = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram))
    return {"architecture": "Zonidra", "vocab": vocab, "width": width, "embedding": emb, "norm": {"eps": eps}, "layers": [dict(e, mlp=f) for e, f in layers]}


CASES = {
    # keys read by several layers behind, unequal windows on the same keys, a layer without a feed-forward
    "all": config([(attention(), moe()), (attention(source=0), dense()), (attention(heads=6, kv_heads=3, dim=16, vdim=8, rot_dims=6, scaling=None, size=40, keep=0), moe(experts=5, identity=3, top=1, shared=0)),
                   (attention(heads=2, size=17, keep=21, source=0), None), (attention(heads=3, kv_heads=3, dim=16, vdim=8, rot_dims=16, base=300.0, size=1, keep=9, source=2), moe(identity=0))]),
    # sizes that no tensor-core kernel takes, one head, windows of a few tokens, a bucket count that is no prime
    "odd": config([(attention(heads=1, kv_heads=1, dim=5, vdim=7, rot_dims=4, size=7, keep=1), dense(ff=13)), (attention(heads=3, kv_heads=1, dim=5, vdim=7, rot_dims=2, size=3, keep=2, source=0), moe(experts=3, identity=1, top=2, ff=5, shared=3)),
                   (attention(heads=3, kv_heads=1, dim=7, vdim=7, rot_dims=2, size=2, keep=5), dense(ff=6))], width=37, vocab=61, bigram=(12, 5, 7)),
    # causal layers, no rotation, wide groups; no pair table
    "causal": config([(attention(heads=6, kv_heads=1, dim=16, vdim=40, rot_dims=0, size=0), dense()), (attention(heads=4, kv_heads=1, dim=32, vdim=40, rot_dims=32, size=64, keep=5), moe(top=7, identity=4))], bigram=None),
    # one bucket and one expert only, no feed-forward at the end
    "narrow": config([(attention(heads=8, kv_heads=8, dim=8, vdim=8, rot_dims=8, size=33, keep=0), moe(experts=1, identity=1, top=2)), (attention(heads=2, kv_heads=1, dim=32, size=20, keep=30), None)],
                     scale=0.7, eps=1e-6, bigram=(1, 3, 4)),
}


def weights(cfg, seed=0, sharp=2.0, dtype=torch.bfloat16):
    """Random tensors (bf16 values) under the checkpoint names. ``sharp`` scales queries and keys, so that single keys stand out of their
    sums; the numbers added to the scores are low enough that most keys weigh little."""
    g = torch.Generator().manual_seed(seed)
    d, out = cfg["width"], {}

    def put(name, *shape, std=None, mean=0.0):
        out[name] = (torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean).to(dtype)

    def unit(name, ff):
        put(name + "gate", ff, d, std=1.5 * d ** -0.5)
        put(name + "up", ff, d, std=1.5 * d ** -0.5)
        put(name + "down", d, ff)

    put("embed", cfg["vocab"], d, std=0.6)
    if cfg["embedding"].get("bigram"):
        put("bigram", cfg["embedding"]["bigram"]["buckets"] + 1, d, std=0.7)
    for i, e in enumerate(cfg["layers"]):
        m, n, L = e["mixer"], f"l{i}.mix.", f"l{i}."
        H, vd = m["heads"], m["vdim"]
        for leaf in ("norm1", "norm1b") + (("norm2", "norm2b") if e["mlp"] else ()):
            put(L + leaf, d, std=0.3, mean=1.0)
        for leaf in ("ls1",) + (("ls2",) if e["mlp"] else ()):
            put(L + leaf, d, std=0.2, mean=0.8)
        out[L + "shift"] = torch.rand(d, generator=g).to(dtype)
        put(n + "q", H * m["dim"], d, std=sharp * d ** -0.5)
        if m.get("kv_from") is None:
            put(n + "k", m["kv_heads"] * m["dim"], d, std=sharp * d ** -0.5)
            put(n + "v", m["kv_heads"] * vd, d)
        put(n + "pb", H, std=1.0, mean=-2.0)
        put(n + "g", H * vd, d)
        put(n + "o", d, H * vd)
        if e["mlp"] and e["mlp"]["kind"] == "dense":
            put(L + "mlp.up", e["mlp"]["ff"], d)
            put(L + "mlp.down", d, e["mlp"]["ff"])
            put(L + "mlp.act", 4, std=0.7)
        elif e["mlp"]:
            r, sh = e["mlp"]["router"], e["mlp"].get("shared")
            put(L + "mlp.router", r["experts"] + r["identity"], d, std=2 * d ** -0.5)
            put(L + "mlp.correction", r["experts"] + r["identity"], std=0.15)
            for x in range(r["experts"]):
                unit(f"{L}mlp.e{x}.", e["mlp"]["expert"]["ff"])
            if sh:
                unit(L + "mlp.shared.", sh["ff"])
                put(L + "mlp.shared.sg", 1, d, std=2 * d ** -0.5)
    put("final.norm", d, std=0.3, mean=1.0)
    put("head", cfg["vocab"], d)
    return out


def oracle(cfg, w, toks):
    return O.forward(cfg, w, toks)


def module_weights(module, w):
    """Fills a mixer or feed-forward module from tensors named like its checkpoint leaves."""
    with torch.no_grad():
        for leaf, t in module.tensors():
            t.copy_(w[leaf])
    return module


def close_routes(cfg, w, toks, margin):
    """Positions of ``toks`` at which some layer's router decides by less than ``margin`` (a rounding may flip such a choice)."""
    seen = []
    real = O.route

    def watch(ww, h, r):
        c = (torch.softmax(h @ ww["router"].T, -1) + ww["correction"]).sort(-1, descending=True)[0]
        if r["top"] < c.shape[1]:
            seen.append(c[:, r["top"] - 1] - c[:, r["top"]] < margin)
        return real(ww, h, r)

    O.route = watch
    try:
        O.forward(cfg, w, toks)
    finally:
        O.route = real
    return torch.stack(seen).any(0) if seen else torch.zeros(len(toks), dtype=torch.bool)


def window_contexts(b, lens, starts, slots, m):
    """Adds to ``b`` the context of its tile-wise portions (``lens`` new tokens behind ``starts`` cached ones; ``slots``: every portion's cache slots
    by position) that a layer with the window of ``m`` reads: tiles of 64 positions that some row sees, and those of the kept tokens."""
    parts, skip = [], []
    for n, s, sl in zip(lens, starts, slots):
        front = -(-m.keep // 64) * 64
        lo = max(0, s - m.window + 1) // 64 * 64
        gone = max(0, lo - front)
        skip.append(gone)
        parts.append(torch.cat([sl[: min(front, s + n)], sl[front + gone : s + n]]))
    cu = torch.tensor([0] + [p.numel() for p in parts]).cumsum(0).to(torch.int32)
    dev = b.positions.device
    b.window_ctx[m.window, m.keep] = (cu.to(dev), torch.cat(parts).to(dev), torch.tensor(skip, dtype=torch.int32, device=dev))
    return b


def standout_case(m, T, bs, far, n, device="cpu", dtype=torch.float32, portion_tiles=False):
    """``n`` new tokens behind ``T - n`` cached ones in scattered pages of a mixer without rotation; to every query key ``far`` weighs about one
    and all others about nothing. Returns (projected rows, batch, key cache, value cache, outputs [n, heads * vdim] by the oracle)."""
    from rl_b200.ops import mixer_ops as X

    g = torch.Generator().manual_seed(far * 100 + n)
    k = torch.zeros(T, m.kv_heads, m.dim)
    k[far, :, 0] = 1.0
    v = torch.randn(T, m.kv_heads, m.vdim, generator=g).to(dtype).float()
    q = torch.zeros(n, m.heads, m.dim)
    q[:, :, 0] = 32.0 / m.scale
    with torch.no_grad():
        m.offset.fill_(-16.0)
    gates = torch.randn(n, m.heads * m.vdim, generator=g).to(dtype).float()
    pages = -(-T // bs)
    order = torch.randperm(pages + 3, generator=g)[:pages]
    kc, vc = (torch.randn(pages + 3, m.kv_heads, bs, w, generator=g) for w in (m.dim, m.vdim))
    t = torch.arange(T)
    slot = order[t // bs] * bs + t % bs
    old = slot[: T - n] if m.kv_from is None else slot
    kc[old // bs, :, old % bs], vc[old // bs, :, old % bs] = k[: old.numel()], v[: old.numel()]
    p = torch.zeros(n, m.in_width)
    p[:, m.q_off : m.q_off + m.heads * m.dim] = q.reshape(n, -1)
    if m.kv_from is None:
        p[:, m.k_off : m.k_off + m.kv_heads * m.dim] = k[T - n :].reshape(n, -1)
        p[:, m.v_off : m.v_off + m.kv_heads * m.vdim] = v[T - n :].reshape(n, -1)
    p[:, m.mix_off : m.mix_off + m.heads * m.vdim] = gates
    pos = torch.arange(T - n, T, dtype=torch.int32)
    bt = torch.zeros(1, pages + 1, dtype=torch.int32)
    bt[0, :pages] = order
    b = X.TokenBatch(ids=None, positions=pos.to(device), slots=slot[T - n :].to(device), n_single=int(n == 1), n_paged=n,
                     block_table=bt.expand(n, -1).contiguous().to(device), seq_lens=(pos + 1).to(device), max_ctx=T)
    if portion_tiles and n > X.PAGED_PORTION:
        cu = torch.tensor([[0, n], [0, T]], dtype=torch.int32, device=device)
        b.n_paged, b.block_table, b.seq_lens, b.whole = 0, b.block_table[:0], b.seq_lens[:0], n == T and m.kv_from is None
        b.cu_q, b.cu_ctx, b.q_tiles, b.ctx_slots = cu[0], cu[1], -(-n // 128), slot.to(device)
        if m.window:
            window_contexts(b, [n], [T - n], [slot], m)
    seen = O.visible(T, {"size": m.window, "keep_first": m.keep} if m.window else None)
    want = torch.zeros(T, m.heads, m.vdim, dtype=torch.float64)
    for h in range(m.heads):
        j = h // (m.heads // m.kv_heads)
        want[:, h] = O.attend(q[:1, h].double().expand(T, -1), k[:, j].double(), v[:, j].double(), m.scale, -16.0, seen)
    want = want[T - n :].reshape(n, -1) * O.sigmoid(gates.double())
    return p.to(device, dtype), b, kc.to(device, dtype), vc.to(device, dtype), want
