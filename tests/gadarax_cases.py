"""Small Gadarax models with random weights for the tests: configuration, tensors, checkpoint folder, engine, oracle logits."""

from __future__ import annotations

import json
import math
import os

import torch

import gadarax_oracle as O
from rl_b200.engine.engine import GenerationEngine
from rl_b200.models.hf_io import load_pretrained


def latent(heads=3, dim=16, rot_dim=8, vdim=24, kv_rank=40, base=10000.0, scaling=None, scale=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
            "scale": scale or (dim + rot_dim) ** -0.5, "rot": {"dims": rot_dim, "base": base, "scaling": scaling} if scaling else {"dims": rot_dim, "base": base}}}


def retention(heads=4, dim=24, vdim=16, rot_dims=None, decay=None, base=10000.0):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or [1 - 2.0 ** -(1 + 2 * i) for i in range(heads)],
            "rot": {"dims": dim if rot_dims is None else rot_dims, "base": base}}}


def config(layers, width=56, vocab=88, loop=None, ff=48, scale=3.5, eps=1e-5):
    """``ff``: MLP width of every layer, or a list with None for layers without one."""
    ffs = ff if isinstance(ff, list) else [ff] * len(layers)
    c = {"architecture": "Gadarax", "vocab": vocab, "width": width, "embedding": {"scale": scale}, "norm": {"eps": eps},
         "layers": [dict(e, mlp={"kind": "dense", "ff": f} if f else None) for e, f in zip(layers, ffs)]}
    return dict(c, loop=loop) if loop else c


YARN = {"factor": 4.0, "original": 48, "fast": 3.0, "slow": 0.4}

CASES = {
    # both mixers, a loop over both kinds, YaRN, unequal sizes
    "loop": config([latent(scaling=YARN), retention(), latent(heads=2, dim=32, rot_dim=16, vdim=8, kv_rank=24), retention(heads=3, dim=8, vdim=40, rot_dims=4)],
                   loop={"start": 1, "stop": 3, "times": 3}, ff=[48, None, 40, 64]),
    # the loop starts at the first layer and ends at the last; no MLP anywhere
    "whole_loop": config([retention(heads=2, dim=16, vdim=16), latent(heads=4, dim=16, rot_dim=8, vdim=8, kv_rank=16)],
                         loop={"start": 0, "stop": 2, "times": 2}, ff=[None, None], width=40),
    # no loop, one pass each; sizes that no tensor-core kernel takes (odd widths), one head
    "odd": config([latent(heads=1, dim=5, rot_dim=6, vdim=7, kv_rank=9), retention(heads=1, dim=7, vdim=5, rot_dims=6, decay=[0.9])],
                  width=37, vocab=61, ff=[13, 11]),
    "attention_only": config([latent(), latent(heads=5, dim=16, rot_dim=24, vdim=16, kv_rank=72)], loop={"start": 0, "stop": 1, "times": 1}),
}


def weights(cfg, seed=0, sharp=2.0):
    """Random tensors (bf16 values) under the checkpoint names. ``sharp`` scales the query and key projections of the attention, so that
    single keys stand out of their sums."""
    g = torch.Generator().manual_seed(seed)
    d = cfg["width"]
    out = {}

    def put(name, *shape, std=None):
        out[name] = (torch.randn(*shape, generator=g) * (std if std is not None else shape[-1] ** -0.5)).to(torch.bfloat16)

    def norm(name, n):
        out[name] = (1 + 0.3 * torch.randn(n, generator=g)).to(torch.bfloat16)

    def dyt(name):
        norm(name, d)
        put(name + ".b", d, std=0.2)
        out[name + ".alpha"] = torch.tensor(0.3 + 0.4 * torch.rand((), generator=g).item()).to(torch.bfloat16)

    put("embed", cfg["vocab"], d, std=0.4)
    if cfg.get("loop"):
        put("loop.step", cfg["loop"]["times"], d, std=0.5)
    for i, e in enumerate(cfg["layers"]):
        m, n = e["mixer"], f"l{i}.mix."
        H = m["heads"]
        dyt(f"l{i}.norm1")
        if e["type"] == "latent_attention":
            put(n + "q", H * (m["dim"] + m["rot_dim"]), d, std=sharp * d ** -0.5)
            put(n + "dkv", m["kv_rank"] + m["rot_dim"], d, std=sharp * d ** -0.5)
            norm(n + "dkv.norm", m["kv_rank"])
            put(n + "uk", H * m["dim"], m["kv_rank"], std=sharp * m["kv_rank"] ** -0.5)
            put(n + "uv", H * m["vdim"], m["kv_rank"])
        else:
            put(n + "q", H * m["dim"], d)
            put(n + "k", H * m["dim"], d)
            put(n + "v", H * m["vdim"], d)
        put(n + "g", H * m["vdim"], d)
        put(n + "o", d, H * m["vdim"])
        if e["mlp"]:
            put(f"l{i}.mlp.up", e["mlp"]["ff"], d)
            put(f"l{i}.mlp.down", d, e["mlp"]["ff"])
    dyt("final.norm")
    return out


def save(cfg, w, path):
    from safetensors.torch import save_file

    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    save_file(w, os.path.join(path, "model.safetensors"))
    return str(path)


def load(cfg, w, path, device="cpu", dtype=torch.float32):
    return load_pretrained(save(cfg, w, path), device=device, dtype=dtype)


def engine(model, pages=24, block_size=16, requests=4, **kw):
    return GenerationEngine(model, block_size=block_size, num_blocks=pages, max_running=requests, max_model_len=pages * block_size,
                            use_cuda_graphs=kw.pop("use_cuda_graphs", False), **kw)


def tokens(cfg, n, seed=0):
    return torch.randint(0, cfg["vocab"], (n,), generator=torch.Generator().manual_seed(100 + seed)).tolist()


def oracle(cfg, w, toks):
    return O.forward(cfg, w, toks)


def gap(got, want):
    """Root mean square difference over the vocabulary (mean taken off) relative to the logits' own spread; worst position."""
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    return (d.pow(2).mean(-1).sqrt() / s.pow(2).mean().sqrt()).max().item() if d.numel() else 0.0


def run_cut(eng, name, toks, cuts, end=True):
    """Logits of every token of one request fed in portions of the given sizes (the last size repeats)."""
    out, at, k = [], 0, 0
    while at < len(toks):
        n = min(cuts[min(k, len(cuts) - 1)], len(toks) - at)
        last = at + n == len(toks)
        out.append(eng.step([(name, toks[at : at + n], list(range(n)))], [name] if (last and end) else [])[0].float().cpu())
        at, k = at + n, k + 1
    return torch.cat(out)


def run_schedule(eng, steps, seqs):
    """``steps``: per step {request: token count}; a request ends with its last token. Returns logits per request."""
    at, out = {}, {}
    for st in steps:
        entries = [(r, seqs[r][at.get(r, 0) : at.get(r, 0) + n], list(range(n))) for r, n in st.items()]
        for r, n in st.items():
            at[r] = at.get(r, 0) + n
        z = eng.step(entries, [r for r in st if at[r] == len(seqs[r])])
        for (r, _, _), zz in zip(entries, z):
            out.setdefault(r, []).append(zz.float().cpu())
    return {r: torch.cat(v) for r, v in out.items()}


def mixed_schedule(lengths, seed=0, live=4):
    """Random mixed batches: portions beside single tokens, requests left out of steps, at most ``live`` at a time."""
    import random

    rng = random.Random(seed)
    left, waiting, running, steps = dict(lengths), list(lengths), [], []
    while waiting or running:
        while waiting and len(running) < live:
            running.append(waiting.pop(0))
        st = {}
        for r in running:
            if rng.random() < 0.25 and len(running) > 1:
                continue
            st[r] = min(left[r], rng.choice([1, 1, 1, 2, 3, 15, 16, 17, 31, 40]))
        for r, n in st.items():
            left[r] -= n
        running = [r for r in running if left[r]]
        if st:
            steps.append(st)
    return steps


def live_pages(steps, block_size):
    """Most pages that the live requests of a schedule hold at once."""
    total, most = {}, 0
    ends = {}
    for i, st in enumerate(steps):
        for r in st:
            ends[r] = i
    for i, st in enumerate(steps):
        for r, n in st.items():
            total[r] = total.get(r, 0) + n
        most = max(most, sum(math.ceil(n / block_size) for n in total.values()))
        for r in [r for r in total if ends[r] == i]:
            del total[r]
    return most
