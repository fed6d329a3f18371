"""Small Kikivik models with random weights for the tests: configuration, tensors, checkpoint folder, oracle logits."""

from __future__ import annotations

import gadarax_cases as G
import kikivik_oracle as O
import torch

engine, tokens, gap, run_cut, run_schedule, mixed_schedule, live_pages, save, load = (
    G.engine, G.tokens, G.gap, G.run_cut, G.run_schedule, G.mixed_schedule, G.live_pages, G.save, G.load)


def attention(heads=4, kv_heads=2, dim=24, vdim=16, rot_dims=16, base=10000.0, factor=3.0, scale=0.3, size=24, v_mix=True):
    rot = {"dims": rot_dims, "base": base}
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": dict(rot, scaling={"factor": factor}) if factor else rot}
    if size:
        m["mask"] = {"size": size}
    return {"type": "attention", "mixer": dict(m, v_mix=True) if v_mix else m}


def latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, q_rank=56, base=5000.0, scale=0.25):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank,
                                                  "scale": scale, "rot": {"dims": rot_dim, "base": base}}}


def dense(ff=44, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=7, top=3, ff=20, shared=28):
    m = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    return dict(m, shared={"ff": shared}) if shared else m


def config(layers, width=56, vocab=88, scale=1.9, eps=1e-4):
    """``layers``: (mixer entry, feed-forward or None) pairs."""
    return {"architecture": "Kikivik", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
            "layers": [dict(e, mlp=f) for e, f in layers]}


CASES = {
    # both mixers and feed-forwards, unequal sizes and chunks, a layer without a feed-forward, one that mixes no values between two that do
    "all": config([(attention(), moe()), (latent(), dense()), (attention(heads=6, kv_heads=3, dim=16, vdim=8, rot_dims=6, factor=0, size=40, v_mix=False), moe(experts=5, top=1, shared=0)),
                   (attention(heads=2, kv_heads=2, dim=20, vdim=16, rot_dims=20, base=300.0, factor=1.5, size=17), None), (latent(heads=5, dim=8, rot_dim=16, vdim=16, kv_rank=24, q_rank=32), moe())]),
    # sizes that no tensor-core kernel takes, one head, rotation of a part, chunks of a few tokens
    "odd": config([(attention(heads=1, kv_heads=1, dim=5, vdim=7, rot_dims=4, size=7), dense(ff=13)), (latent(heads=1, dim=3, rot_dim=2, vdim=5, kv_rank=9, q_rank=11), moe(experts=3, top=2, ff=5, shared=3)),
                   (attention(heads=3, kv_heads=1, dim=7, vdim=7, rot_dims=2, factor=0, size=3), dense(ff=6, limit=0.4))], width=37, vocab=61),
    # attention alone, wide groups, no rotation, no chunks in one layer
    "attention_only": config([(attention(heads=6, kv_heads=1, dim=16, vdim=40, rot_dims=0, factor=0, size=0), dense()), (attention(heads=4, kv_heads=1, dim=32, vdim=40, rot_dims=32, size=64), moe(top=7))]),
    "latent_only": config([(latent(heads=8, vdim=8), moe(experts=12, top=1)), (latent(heads=2, dim=32, rot_dim=24, kv_rank=16, q_rank=24), None)], scale=0.7, eps=1e-6),
}


def weights(cfg, seed=0, sharp=2.0, dtype=torch.bfloat16):
    """Random tensors (bf16 values) under the checkpoint names. ``sharp`` scales queries and keys, so that single keys stand out of their
    sums; gate and up rows are large enough to meet their limits, experts' weights differ much between tokens."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    out = {}

    def put(name, *shape, std=None, mean=0.0):
        out[name] = (torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5) + mean).to(dtype)

    def norm(name, n, size=1.0):
        put(name, n, std=0.3 * size, mean=size)

    def glu(name, ff):
        put(name + "gate", ff, d, std=1.5 * d ** -0.5)
        put(name + "up", ff, d, std=1.5 * d ** -0.5)
        put(name + "down", d, ff)

    put("embed", cfg["vocab"], d, std=0.6)
    for i, e in enumerate(cfg["layers"]):
        m, n = e["mixer"], f"l{i}.mix."
        H, vd = m["heads"], m["vdim"]
        norm(f"l{i}.norm1", d)
        if e["type"] == "attention":
            for leaf, r in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * vd)):
                put(n + leaf, r, d)
            norm(n + "q.norm", m["dim"], sharp ** 0.5)
            norm(n + "k.norm", m["dim"], sharp ** 0.5)
            if m.get("v_mix"):
                out[n + "vmix"] = torch.tensor(0.2 + 0.6 * torch.rand((), generator=g).item()).to(dtype)
        else:
            put(n + "dq", m["q_rank"], d)
            norm(n + "dq.norm", m["q_rank"])
            put(n + "uq", H * (m["dim"] + m["rot_dim"]), m["q_rank"], std=sharp * m["q_rank"] ** -0.5)
            put(n + "dkv", m["kv_rank"] + m["rot_dim"], d, std=sharp * d ** -0.5)
            norm(n + "dkv.norm", m["kv_rank"])
            put(n + "uk", H * m["dim"], m["kv_rank"])
            put(n + "uv", H * vd, m["kv_rank"])
        put(n + "o", d, H * vd)
        if e["mlp"]:
            norm(f"l{i}.norm2", d)
            if e["mlp"]["kind"] == "dense":
                glu(f"l{i}.mlp.", e["mlp"]["ff"])
            else:
                E = e["mlp"]["router"]["experts"]
                put(f"l{i}.mlp.router", E, d, std=2 * d ** -0.5)
                for x in range(E):
                    glu(f"l{i}.mlp.e{x}.", e["mlp"]["expert"]["ff"])
                if e["mlp"].get("shared"):
                    glu(f"l{i}.mlp.shared.", e["mlp"]["shared"]["ff"])
    norm("final.norm", d)
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
        s = O.sigmoid(h @ ww["router"].T).sort(-1, descending=True)[0]
        if r["top"] < r["experts"]:
            seen.append(s[:, r["top"] - 1] - s[:, r["top"]] < margin)
        return real(ww, h, r)

    O.route = watch
    try:
        O.forward(cfg, w, toks)
    finally:
        O.route = real
    return torch.stack(seen).any(0) if seen else torch.zeros(len(toks), dtype=torch.bool)


def standout_case(mixer, T, bs, far, n, device="cpu", dtype=torch.float32, portion_tiles=False):
    """``n`` new tokens behind ``T - n`` cached ones in scattered pages of a grouped attention ``mixer`` without rotation; every query scores key
    ``far`` far above all others. Returns (projected rows, batch, key cache, value cache, outputs [n, heads * vdim] by the oracle)."""
    from rl_b200.ops import mixer_ops as X

    m = mixer
    g = torch.Generator().manual_seed(far * 100 + n)
    k = torch.full((T, m.kv_heads, m.dim), 0.1)
    k[:, :, 0] = 0.0                # (exactly: rounding must not tell the other keys apart)
    k[far, :, 0] = 1.0
    v = torch.randn(T, m.kv_heads, m.vdim, generator=g)
    q = torch.zeros(n, m.heads, m.dim)
    q[:, :, 0] = 30.0
    eps = m.eps
    kn, qn = O.rms(k.double(), eps), O.rms(q.double(), eps)
    pages = -(-T // bs)
    order = torch.randperm(pages + 3, generator=g)[:pages]
    kc, vc = (torch.randn(pages + 3, m.kv_heads, bs, w, generator=g) for w in (m.dim, m.vdim))
    t = torch.arange(T)
    slot = order[t // bs] * bs + t % bs
    kc[slot[: T - n] // bs, :, slot[: T - n] % bs], vc[slot[: T - n] // bs, :, slot[: T - n] % bs] = kn[: T - n].float(), v[: T - n]
    p = torch.zeros(n, m.in_width)
    p[:, m.q_off : m.q_off + m.heads * m.dim] = q.reshape(n, -1)
    p[:, m.k_off : m.k_off + m.kv_heads * m.dim] = k[T - n :].reshape(n, -1)
    p[:, m.v_off : m.v_off + m.kv_heads * m.vdim] = v[T - n :].reshape(n, -1)
    pos = torch.arange(T - n, T, dtype=torch.int32)
    bt = torch.zeros(1, pages + 1, dtype=torch.int32)
    bt[0, :pages] = order
    b = X.TokenBatch(ids=None, positions=pos.to(device), slots=slot[T - n :].to(device), n_single=int(n == 1), n_paged=n,
                     block_table=bt.expand(n, -1).contiguous().to(device), seq_lens=(pos + 1).to(device), max_ctx=T)
    if portion_tiles and n > X.PAGED_PORTION:
        lo = (T - n) // m.chunk * m.chunk if m.chunk else 0
        cu = torch.tensor([[0, n], [0, T], [0, T - lo]], dtype=torch.int32, device=device)
        b.n_paged, b.block_table, b.seq_lens, b.whole = 0, b.block_table[:0], b.seq_lens[:0], n == T
        b.cu_q, b.cu_ctx, b.q_tiles, b.ctx_slots = cu[0], cu[1], -(-n // 128), slot.to(device)
        if m.chunk:
            b.chunk_ctx[m.chunk] = (cu[2], slot[lo:].to(device), lo == T - n)
    seen = O.visible(T, m.chunk or None)
    want = torch.zeros(T, m.heads, m.vdim, dtype=torch.float64)
    for h in range(m.heads):
        j = h // (m.heads // m.kv_heads)
        want[:, h] = O.attend(torch.cat([qn[:1, h].expand(T - n, -1), qn[:, h]]), kn[:, j], v[:, j].to(dtype).double(), m.scale, seen)
    return p.to(device, dtype), b, kc.to(device, dtype), vc.to(device, dtype), want[T - n :].reshape(n, -1)
