"""Small Redarax models with random weights for the tests: configuration, tensors, checkpoint folder, oracle logits."""

from __future__ import annotations

import gadarax_cases as G
import redarax_oracle as O
import torch

engine, tokens, gap, run_cut, run_schedule, mixed_schedule, live_pages, save, load = (
    G.engine, G.tokens, G.gap, G.run_cut, G.run_schedule, G.mixed_schedule, G.live_pages, G.save, G.load)


def attention(heads=4, kv_heads=2, dim=24, vdim=16, rot_dims=16, base=10000.0, scale=0.3):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": {"dims": rot_dims, "base": base}}}


def mamba2(heads=6, vdim=12, state=20, groups=3, norm_groups=2, conv=3):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv}}


def delta(heads=4, kv_heads=2, dim=20, vdim=28, conv=4):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv}}


def dense(ff=44, limit=1.2):
    return {"kind": "dense", "ff": ff, "limit": limit}


def moe(experts=8, top=3, ff=20, limit=0.9, groups=(4, 2)):
    r = {"experts": experts, "top": top}
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": dict(r, groups={"count": groups[0], "keep": groups[1]}) if groups else r}


def config(layers, width=56, vocab=88, side=12, mult=0.6, scale=1.7, cap=9.0, eps=1e-5):
    """``layers``: (mixer entry, feed-forward or None) pairs."""
    c = {"architecture": "Redarax", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "logit_scale": scale, "logit_softcap": cap,
         "layers": [dict(e, mlp=f) for e, f in layers]}
    return dict(c, token_side={"dim": side}) if side else c


CASES = {
    # every mixer and both feed-forwards, unequal sizes, one layer without a feed-forward
    "all": config([(mamba2(), moe()), (delta(), dense()), (attention(), moe(experts=6, top=2, groups=(2, 1))), (delta(heads=3, kv_heads=3, dim=8, vdim=40, conv=2), None)]),
    # sizes that no tensor-core kernel takes, one head, one tap, no rotation, no groups, no token input
    "odd": config([(attention(heads=1, kv_heads=1, dim=5, vdim=7, rot_dims=0), dense(ff=13)), (mamba2(heads=1, vdim=7, state=5, groups=1, norm_groups=1, conv=1), moe(experts=5, top=1, ff=3, groups=None)),
                   (delta(heads=2, kv_heads=1, dim=7, vdim=5, conv=1), dense(ff=6))], width=37, vocab=61, side=0),
    # attention alone (pages are shared between equal prompts), wide groups, a token input of odd width
    "attention_only": config([(attention(heads=6, kv_heads=1, dim=16, vdim=40, rot_dims=2), dense()), (attention(heads=4, kv_heads=4, dim=32, vdim=8, rot_dims=32), moe(groups=(1, 1)))], side=5, cap=0.0),
    # recurrent alone; a state of many taps
    "recurrent_only": config([(delta(heads=6, kv_heads=2, conv=6), None), (mamba2(heads=8, vdim=8, groups=2, norm_groups=8, conv=5), dense())], mult=1.0, scale=1.0),
}


def weights(cfg, seed=0, sharp=2.0, dtype=torch.bfloat16):
    """Random tensors (bf16 values) under the checkpoint names. ``sharp`` scales the query and key norms of the attention, so that single keys
    stand out of their sums; gate and up rows are large enough to meet their limits, decays range from quick to slow."""
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

    put("embed", cfg["vocab"], d, std=1.0)
    n_side = cfg["token_side"]["dim"] if cfg.get("token_side") else 0
    if n_side:
        put("side.embed", cfg["vocab"], len(cfg["layers"]) * n_side, std=1.0)
    for i, e in enumerate(cfg["layers"]):
        m, n = e["mixer"], f"l{i}.mix."
        H, vd = m["heads"], m["vdim"]
        norm(f"l{i}.norm1", d)
        if e["type"] == "attention":
            for leaf, r in (("q", H * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", m["kv_heads"] * vd)):
                put(n + leaf, r, d)
                put(n + leaf + ".b", r, std=0.5)
            norm(n + "q.norm", m["dim"], sharp ** 0.5)
            norm(n + "k.norm", m["dim"], sharp ** 0.5)
            put(n + "o.b", d, std=0.3)
        elif e["type"] == "mamba2":
            C = H * vd + 2 * m["groups"] * m["state"]
            put(n + "in", H * vd + C + H, d)
            put(n + "conv", C, m["conv"], std=0.6)
            put(n + "conv.b", C, std=0.3)
            put(n + "dt_bias", H, std=1.0, mean=-1.5)
            put(n + "A_log", H, std=0.8)
            put(n + "D", H, std=0.5, mean=1.0)
            norm(n + "norm", H * vd)
        else:
            for leaf, r in (("q", m["kv_heads"] * m["dim"]), ("k", m["kv_heads"] * m["dim"]), ("v", H * vd)):
                put(n + leaf, r, d)
                put(n + leaf + ".conv", r, m["conv"], std=0.6)
            put(n + "g", H * vd, d)
            put(n + "b", H, d, std=2 * d ** -0.5)
            put(n + "a", H, d)
            put(n + "A_log", H, std=0.8, mean=-0.5)
            put(n + "dt_bias", H, std=1.0, mean=-1.5)
            norm(n + "norm", vd)
        put(n + "o", d, H * vd)
        if e["mlp"]:
            norm(f"l{i}.norm2", d)
            if e["mlp"]["kind"] == "dense":
                glu(f"l{i}.mlp.", e["mlp"]["ff"])
            else:
                E = e["mlp"]["router"]["experts"]
                put(f"l{i}.mlp.router", E, d, std=2 * d ** -0.5)
                put(f"l{i}.mlp.correction", E, std=0.4, mean=-0.5)      # choice scores of both signs
                for x in range(E):
                    glu(f"l{i}.mlp.e{x}.", e["mlp"]["expert"]["ff"])
        if n_side:
            put(f"l{i}.side.gate", n_side, d)
            put(f"l{i}.side.proj", d, n_side)
            norm(f"l{i}.side.norm", d)
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
        s = O.sigmoid(h @ ww["router"].T) + ww["correction"]
        gr = r.get("groups") or {"count": 1, "keep": 1}
        size = r["experts"] // gr["count"]
        bad = torch.zeros(h.shape[0], dtype=torch.bool)
        for t in range(h.shape[0]):
            c = s[t].view(gr["count"], size)
            gs = c.topk(min(2, size), -1)[0].sum(-1).sort(descending=True)
            if gr["keep"] < gr["count"]:
                bad[t] |= bool(gs[0][gr["keep"] - 1] - gs[0][gr["keep"]] < margin)
            e = c[gs[1][: gr["keep"]]].reshape(-1).sort(descending=True)[0]
            if r["top"] < e.numel():
                bad[t] |= bool(e[r["top"] - 1] - e[r["top"]] < margin)
        seen.append(bad)
        return real(ww, h, r)

    O.route = watch
    try:
        O.forward(cfg, w, toks)
    finally:
        O.route = real
    return torch.stack(seen).any(0) if seen else torch.zeros(len(toks), dtype=torch.bool)
