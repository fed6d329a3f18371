"""Serving throughput of layer-list models beside the framework's closest model at equal size (Gadarax: the Llama architecture, Redarax and
Kikivik: Qwen3-MoE, Zonidra: Kikivik), and the kernels' distance from their rooflines beside the like kernels of the closest path.

    python bench.py --config gadarax-serving | redarax-serving | kikivik-serving | zonidra-serving [--steps K --warmup W]

Random weights, random prompts. Whole-model figures come from ``GenerationEngine``: prefill of packed prompts (device time of the
forward pass) and decoding through the captured step (device time of the graph replays). Kernel figures are CUDA-event times of a
captured graph that runs the operator over buffer sets larger than L2 together.
"""

from __future__ import annotations

import json
import math
import os

import torch

from rl_b200.engine.engine import GenerationEngine, SamplingParams
from rl_b200.models.config import ModelConfig, preset
from rl_b200.models.transformer import build_model
from rl_b200.ops import engine_ops as E
from rl_b200.ops import functional as F
from rl_b200.ops import lib as L
from rl_b200.ops import mixer_ops as X

SIZES = {   # (preset, Llama twin: same width and run count, MHA with 128-wide heads, MLP sized to equal weights per layer run)
    "gadarax-1b": dict(hidden_size=2048, num_attention_heads=16),
    "gadarax-4b": dict(hidden_size=4096, num_attention_heads=32),
}
REDARAX = ("redarax-2b", "redarax-7b")
KIKIVIK = ("kikivik-2b", "kikivik-7b")
ZONIDRA = ("zonidra-2b", "zonidra-7b")
PREFILL = ((1, 4096), (8, 1024))      # (prompts, tokens each)
DECODE = ((16, 4096), (64, 2048))     # (sequences, context)


def llama_twin(name: str) -> ModelConfig:
    """Llama-architecture model of the same width, the same number of layer runs and the same weight bytes streamed per token."""
    c = preset(name)
    base = SIZES[name]
    d, runs = c.hidden_size, c.layer_runs
    per_run = []
    for i, _ in runs:
        m, ff = c.mixers[i]["mixer"], c.mixers[i]["mlp"]["ff"]
        H, kd, vd = m["heads"], m["dim"], m["vdim"]
        if c.mixers[i]["type"] == "latent_attention":
            per_run.append(d * (H * (kd + m["rot_dim"]) + m["kv_rank"] + m["rot_dim"] + 2 * H * vd) + H * (kd + vd) * m["kv_rank"] + 2 * d * ff)
        else:
            per_run.append(d * (2 * H * kd + 3 * H * vd) + 2 * d * ff)
    mean = sum(per_run) / len(per_run)
    ff = round((mean - 4 * d * d) / (3 * d) / 128) * 128
    return ModelConfig(model_type="llama", vocab_size=c.vocab_size, intermediate_size=ff, num_hidden_layers=len(runs), head_dim=128,
                       num_key_value_heads=base["num_attention_heads"], rms_norm_eps=1e-5, rope_theta=500000.0, tie_word_embeddings=True, **base)


def moe_twin(name: str) -> ModelConfig:
    """Qwen3-MoE model of the same width, layers, attention heads, experts and choice, the experts' width set for the same number of weights."""
    c = preset(name)
    att = next(e["mixer"] for e in c.mixers if e["type"] == "attention")
    r = next(e["mlp"]["router"] for e in c.mixers if e["mlp"] and e["mlp"]["kind"] == "moe")
    t = ModelConfig(model_type="qwen3_moe", vocab_size=c.vocab_size, hidden_size=c.hidden_size, intermediate_size=c.intermediate_size,
                    num_hidden_layers=c.num_hidden_layers, num_attention_heads=att["heads"], num_key_value_heads=att["kv_heads"], head_dim=att["dim"],
                    rms_norm_eps=1e-6, rope_theta=1e6, qk_norm=True, num_experts=r["experts"], num_experts_per_tok=r["top"], moe_intermediate_size=0)
    per = c.num_hidden_layers * r["experts"] * 3 * c.hidden_size
    t.moe_intermediate_size = round((c.num_parameters() - t.num_parameters()) / per / 64) * 64
    return t


def kikivik_twin(name: str) -> ModelConfig:
    """Kikivik model of the same width, layers, attention heads, experts and choice: chunks as long as the window, gated units of the same number of
    weights, the experts' width set for the same number of weights altogether."""
    c = preset(name)
    layers = []
    for e in c.mixers:
        m, mlp = {k: v for k, v in e["mixer"].items() if k != "kv_from"}, e["mlp"]
        m.update(mask={"size": m["mask"]["size"]}, rot={"dims": m["dim"], "base": 1e6, "scaling": {"factor": 4.0}}, v_mix=True)
        if mlp["kind"] == "dense":
            mlp = {"kind": "dense", "ff": round(mlp["ff"] * 2 / 3 / 64) * 64, "limit": 7.0}
        else:
            mlp = {"kind": "moe", "expert": dict(mlp["expert"]), "router": {"experts": mlp["router"]["experts"], "top": mlp["router"]["top"]}, "shared": dict(mlp["shared"])}
        layers.append({"type": "attention", "mixer": m, "mlp": mlp})
    hf = {"architecture": "Kikivik", "vocab": c.vocab_size, "width": c.hidden_size, "embedding": {"scale": 2.0}, "norm": {"eps": 1e-6}, "layers": layers}
    moe = [e["mlp"] for e in layers if e["mlp"]["kind"] == "moe"]
    per = sum(m["router"]["experts"] * 3 * c.hidden_size for m in moe)
    more = c.num_parameters() - c.bigram["buckets"] * c.hidden_size - ModelConfig.from_hf_dict(hf).num_parameters()      # (of the pair table a few rows are read)
    for m in moe:
        m["expert"]["ff"] += round(more / per / 8) * 8
    return ModelConfig.from_hf_dict(hf)


def timed(fn, steps: int, warmup: int) -> float:
    """Mean ms per call, CUDA events around ``steps`` calls after ``warmup``."""
    for _ in range(warmup):
        fn()
    torch.cuda.synchronize()
    a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    a.record()
    for _ in range(steps):
        fn()
    b.record()
    torch.cuda.synchronize()
    return a.elapsed_time(b) / steps


def timed_graph(fns, steps: int = 5, warmup: int = 3) -> float:
    """Mean ms per operator call: ``fns`` (the operator over different buffers, together larger than L2) captured one after another."""
    side = torch.cuda.Stream()
    side.wait_stream(torch.cuda.current_stream())
    with torch.cuda.stream(side):
        for f in fns:
            f()
    torch.cuda.current_stream().wait_stream(side)
    torch.cuda.synchronize()
    g = torch.cuda.CUDAGraph()
    with torch.cuda.graph(g):
        for f in fns:
            f()
    return timed(g.replay, steps, warmup) / len(fns)


def engine_for(cfg: ModelConfig, tokens: int, seqs: int, max_len: int):
    model = build_model(cfg, device="cuda", dtype=torch.bfloat16, seed=0)
    return GenerationEngine(model, block_size=64, num_blocks=tokens // 64 + 2 * seqs + 2, max_running=seqs, max_model_len=max_len, max_prefill_tokens=16384,
                            enable_prefix_caching=False)


def prefill_ms(eng, n: int, length: int, steps: int, warmup: int) -> float:
    g = torch.Generator().manual_seed(1)
    eng.wake()
    items = []
    for j in range(n):
        toks = torch.randint(0, eng.cfg.vocab_size, (length,), generator=g).tolist()
        eng.sched.open(j)
        eng.sched.extend(j, length)
        if eng.stateful:
            eng._state_row[j] = eng._free_rows.pop()
        items.append((j, toks, 0, length))
    if eng.mixer:     # the forward pass alone: batch tensors are built once
        b, _ = eng._token_batch([(sid, t, 0) for sid, t, _, _ in items])
        rows = torch.arange(1, n + 1, device="cuda") * length - 1
        ms = timed(lambda: eng._mixer_forward(b, rows), steps, warmup)
    else:
        from rl_b200.models.transformer import PackedBatch

        ids = torch.tensor([t for _, ts, _, _ in items for t in ts], dtype=torch.int32, device="cuda")
        cu = torch.arange(0, n + 1, dtype=torch.int32, device="cuda") * length
        batch = PackedBatch(ids, torch.arange(length, dtype=torch.int32, device="cuda").repeat(n), cu, length)
        slots = torch.cat([eng.sched.slots(j, 0, length) for j in range(n)]).cuda()
        ms = timed(lambda: eng._prefill_forward(batch, slots, (cu[1:] - 1).long()), steps, warmup)
    for j in range(n):
        eng.sched.close(j)
        if eng.stateful:
            eng._free_rows.append(eng._state_row.pop(j))
    return ms


def decode_ms(eng, n: int, ctx: int, steps: int, warmup: int) -> float:
    """Device time of one captured decode step (forward, sampling, advance) at about ``ctx`` cached tokens per sequence."""
    eng.wake()
    st = eng._static_buffers()
    B = eng._bucket(n)
    eng._n_stop = 0
    per = ctx // 64
    perm = torch.randperm(eng.num_blocks)[: n * per].to(torch.int32)
    st["block_table"].zero_()
    st["block_table"][:n, :per] = perm.view(n, per).cuda()
    st["win_step"].zero_()
    st["active"].fill_(0)
    st["state_rows"][:n] = torch.arange(1, n + 1, device="cuda")
    sp = SamplingParams(greedy=True, max_new_tokens=1)

    def reset():     # the same step every time: the last token of each sequence
        st["ids"][:n] = 5
        st["positions"][:n] = ctx - 1
        st["seq_lens"][:n] = ctx
        st["slots"][:n] = (st["block_table"][:n, per - 1].long() * 64 + 63)

    prev = E.skinny_static_weights(True)
    splits = E.choose_splits(B, eng.hkv, max(eng.max_model_len // 2, 1), 64, eng._sm_count)
    no, nml = E.decode_scratch_sizes(B, eng.hq, splits, eng.cfg.head_dim)
    scratch = (torch.empty(no, dtype=torch.float32, device="cuda"), torch.empty(nml, dtype=torch.float32, device="cuda")) if splits > 1 else None
    reset()
    with torch.no_grad():
        ms = timed_graph([lambda: eng._decode_body(st, B, sp, splits, scratch)], max(steps, 10), warmup)
    E.skinny_static_weights(bool(prev))
    return ms


def peaks() -> dict:
    path = os.path.join(os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__)))), "MEASURED_PEAKS.json")
    try:
        p = json.load(open(path))
        return dict(hbm=p["hbm_gbs"] * 1e9, flops=p["bf16_tflops"] * 1e12, of="measured")
    except OSError:
        return dict(hbm=6.65e12, flops=1.59e15, of="fallback")


def kernel_table(name: str) -> list:
    """[(kernel, ms, roofline ms, fraction of roofline)] of the operators at the preset's sizes, each followed by the like kernel of the
    Llama path (marked 'like:')."""
    pk = peaks()
    c = preset(name)
    model = build_model(c, device="cuda", dtype=torch.bfloat16, seed=0)
    att = next(l for l in model.layers if l.mixer.kind == "latent_attention")
    ret = next(l for l in model.layers if l.mixer.kind == "retention")
    d = c.hidden_size
    dev, bf = "cuda", torch.bfloat16
    out = []

    def add(label, ms, flops=0.0, nbytes=0.0):
        roof = max(flops / pk["flops"], nbytes / pk["hbm"]) * 1e3
        out.append(dict(kernel=label, ms=round(ms, 4), roofline_ms=round(roof, 4), fraction=round(roof / ms, 3)))

    with torch.no_grad():
        # products (decode and prefill rows)
        for T in (64, 4096):
            for label, layer in (("in_proj attention layer", att), ("out_proj attention layer", att)):
                w = layer.in_proj if label.startswith("in") else layer.out_proj
                N, K = w.shape
                nb = 2 * (N * K + T * (N + K)) + (8 * T * N if label.startswith("out") else 0)
                sets = copies(lambda: (torch.randn(T, K, device=dev).to(bf), w.detach().clone(), torch.randn(T, N, device=dev) if label.startswith("out") else None), nb)
                if label.startswith("in"):
                    ms = timed_graph([lambda s=s: X.in_proj(s[0], s[1], layer.up_off) for s in sets])
                else:
                    ms = timed_graph([lambda s=s: X.out_proj_(s[2], s[0], s[1], None, None, layer.norm) for s in sets])
                add(f"{label}, {T} rows", ms, 2.0 * T * N * K, nb)
                plain = timed_graph([lambda s=s: F.gemm(s[0], s[1]) for s in sets])
                add(f"like: plain GEMM, {T} rows", plain, 2.0 * T * N * K, 2 * (N * K + T * (N + K)))
                del sets
        # decode attention
        m = att.mixer
        for n, ctx in DECODE:
            b = rows_batch(n, ctx)
            nb = n * ctx * m.latent_width * 2 + m.kv_up.numel() * 2
            sets = copies(lambda: (torch.randn(n, att.in_width, device=dev).to(bf), torch.randn(n * ctx // 64, 64, m.latent_width, device=dev).to(bf)), nb)
            add(f"latent attention decode (all kernels), {n} x {ctx}", timed_graph([lambda s=s: X.latent_attention_(s[0], m, b, s[1]) for s in sets]),
                2.0 * n * ctx * m.heads * (2 * m.rank + m.rot_dim), nb)
            del sets
            H = m.heads
            nb = n * ctx * H * 128 * 2 * 2
            sets = copies(lambda: (torch.randn(n, 3 * H * 128, device=dev).to(bf), torch.randn(n * ctx // 64, H, 64, 128, device=dev).to(bf),
                                   torch.randn(n * ctx // 64, H, 64, 128, device=dev).to(bf)), nb)
            sp = E.choose_splits(n, H, ctx // 2, 64)
            add(f"like: paged decode attention, {n} x {ctx}", timed_graph([lambda s=s: E.paged_decode(s[0], s[1], s[2], b.block_table, b.seq_lens, H, H, 128,
                                                                                                   num_splits=sp) for s in sets]), 4.0 * n * ctx * H * 128, nb)
            del sets
        # prefill attention
        for n, length in PREFILL:
            b = portion_batch(n, length)
            T = n * length
            pairs = n * length * length / 2
            cache = torch.zeros((T // 64, 64, m.latent_width), dtype=bf, device=dev)
            nb = 2 * T * (att.in_width + 2 * m.heads * (m.dim + m.vdim))
            sets = copies(lambda: torch.randn(T, att.in_width, device=dev).to(bf), nb)
            fl = 2.0 * pairs * m.heads * (m.dim + m.rot_dim + m.vdim) + 2.0 * T * m.kv_up.numel()
            add(f"latent attention prefill (all kernels), {n} x {length}", timed_graph([lambda s=s: X.latent_attention_(s, m, b, cache) for s in sets]), fl, nb)
            H = m.heads
            sets = copies(lambda: torch.randn(T, 3 * H * 128, device=dev).to(bf), nb)
            add(f"like: flash attention, {n} x {length}", timed_graph([lambda s=s: F.attention_varlen(s, b.cu_q, length, H, H, 128) for s in sets]),
                4.0 * pairs * H * 128, 2 * T * 4 * H * 128)
            del sets
        # retention
        r = ret.mixer
        for n, _ in DECODE:
            b = rows_batch(n, 64)
            nb = n * r.heads * r.dim * r.vdim * 8
            sets = copies(lambda: (torch.randn(n, ret.in_width, device=dev).to(bf), torch.randn(n, r.heads, r.dim, r.vdim, device=dev)), nb)
            add(f"retention decode, {n} rows", timed_graph([lambda s=s: X.retention_(s[0], r, b, s[1]) for s in sets]), 0.0, nb)
            del sets
        for n, length in PREFILL:
            b = portion_batch(n, length)
            T, C = n * length, X.CHUNK
            S = torch.zeros((n, r.heads, r.dim, r.vdim), device=dev)
            nb = 2 * T * r.heads * (3 * r.dim + 3 * r.vdim) + (T // C) * r.heads * r.dim * r.vdim * 16
            fl = 2.0 * T * r.heads * (C / 2 * (r.dim + r.vdim) + 2 * r.dim * r.vdim)
            sets = copies(lambda: torch.randn(T, ret.in_width, device=dev).to(bf), 2 * T * ret.in_width)
            add(f"retention prefill (all kernels), {n} x {length}", timed_graph([lambda s=s: X.retention_(s, r, b, S) for s in sets]), fl, nb)
            del sets
        mc = ModelConfig(model_type="nemotron_h", vocab_size=64, hidden_size=d, intermediate_size=64, num_hidden_layers=1, layers_block_type=["mamba"],
                         num_attention_heads=1, num_key_value_heads=1, head_dim=64, use_rope=False, mlp_gated=False, mamba_num_heads=r.heads,
                         mamba_head_dim=r.vdim, ssm_state_size=r.dim, mamba_n_groups=r.heads, mamba_chunk_size=128)
        from rl_b200.models.mamba import ssd_scan, ssd_step

        A = -torch.rand(r.heads, device=dev)
        n, length = PREFILL[1]
        x, dt = torch.randn(n, length, r.heads, r.vdim, device=dev), torch.rand(n, length, r.heads, device=dev) * 0.1
        Bm, Cm = torch.randn(n, length, r.heads, r.dim, device=dev), torch.randn(n, length, r.heads, r.dim, device=dev)
        T = n * length
        add(f"like: Mamba-2 scan, {n} x {length}", timed(lambda: ssd_scan(x, dt, A, Bm, Cm, 128), 3, 2), 2.0 * T * r.heads * (64 * (r.dim + r.vdim) + 2 * r.dim * r.vdim),
            4 * T * r.heads * (2 * r.dim + 2 * r.vdim) + (T // 128) * r.heads * r.dim * r.vdim * 16)
        n = DECODE[1][0]
        S = torch.randn(n, r.heads, r.vdim, r.dim, device=dev)
        add(f"like: Mamba-2 step, {n} rows", timed(lambda: ssd_step(x[:1, :n].transpose(0, 1)[:, 0], dt[0, :n], A, Bm[0, :n], Cm[0, :n], S), 5, 3), 0.0, S.numel() * 8)
        del mc
    return out


def copies(make, nbytes):
    """Buffer sets that together are larger than L2."""
    return [make() for _ in range(max(2, min(24, math.ceil(200e6 / max(1, nbytes)))))]


def rows_batch(n, ctx, dev="cuda"):
    pages = ctx // 64
    bt = torch.arange(n * pages, dtype=torch.int32, device=dev).view(n, pages)
    pos = torch.full((n,), ctx - 1, dtype=torch.int32, device=dev)
    return X.TokenBatch(ids=None, positions=pos, slots=bt[:, -1].long() * 64 + 63, n_single=n, n_paged=n, block_table=bt, seq_lens=pos + 1,
                        state_rows=torch.arange(n, device=dev), max_ctx=ctx)


def portion_batch(n, length, dev="cuda"):
    T, pages = n * length, length // 64
    cu = torch.arange(n + 1, dtype=torch.int32, device=dev) * length
    pos = torch.arange(length, dtype=torch.int32, device=dev).repeat(n)
    pc, cr, cn = (t.to(dev) for t in X.chunk_lists([length] * n))
    return X.TokenBatch(ids=None, positions=pos, slots=torch.arange(T, device=dev), n_single=0, n_paged=0, seq_lens=pos[:0],
                        block_table=torch.zeros((0, pages), dtype=torch.int32, device=dev), state_rows=torch.arange(n, device=dev), cu=cu, piece_chunk=pc,
                        chunk_row=cr, chunk_rows=cn, cu_q=cu, cu_ctx=cu, ctx_slots=torch.arange(T, device=dev), q_tiles=n * -(-length // 128), whole=True,
                        row_off=pos, row_state=torch.arange(n, device=dev).repeat_interleave(length))


def redarax_table(name: str) -> list:
    """``kernel_table`` of a post-norm layer-list preset."""
    from rl_b200.models.mixers import RetentionMixer
    from rl_b200.models.moe import MoEMLP
    from rl_b200.ops import layer_ops as Y
    from rl_b200.ops import sequence_ops as S

    pk, c, dev, bf = peaks(), preset(name), "cuda", torch.bfloat16
    model = build_model(c, device=dev, dtype=bf, seed=0)
    pick = lambda kind: next(l for l in model.layers if l.mixer.kind == kind)   # noqa: E731
    d, out = c.hidden_size, []

    def add(label, ms, flops=0.0, nbytes=0.0):
        roof = max(flops / pk["flops"], nbytes / pk["hbm"]) * 1e3
        out.append(dict(kernel=label, ms=round(ms, 4), roofline_ms=round(roof, 4), fraction=round(roof / ms, 3)))

    rows = lambda T, n: torch.randn(T, n, device=dev).to(bf)   # noqa: E731
    with torch.no_grad():
        # products with what follows them
        dl, at = pick("delta"), pick("attention")
        glu = next(l.ff for l in model.layers if l.ff is not None and not hasattr(l.ff, "router"))
        for T in (64, 4096):
            for label, w, bias, lim in (("delta in_proj", dl.mixer.in_proj, None, None), ("attention in_proj + bias", at.mixer.in_proj, at.mixer.in_bias, None),
                                        ("out_proj", dl.mixer.out_proj, None, None), ("gate_up + clamped unit", glu.gate_up, None, glu.limit)):
                N, K = w.shape
                nb = 2 * (N * K + T * (K + (N if lim is None else N // 2)))
                sets = copies(lambda: (rows(T, K), w.detach().clone()), nb)
                add(f"{label} [{N} x {K}], {T} rows", timed_graph([lambda s=s: Y.linear(s[0], s[1], bias, lim) for s in sets]), 2.0 * T * N * K, nb)
                add("like: plain GEMM", timed_graph([lambda s=s: F.gemm(s[0], s[1]) for s in sets]), 2.0 * T * N * K, 2 * (N * K + T * (N + K)))
                del sets
            # the join beside the residual add + RMS norm of the closest model
            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d), rows(T, d)), 12 * T * d)
            add(f"join: x += m norm(y), {T} rows", timed_graph([lambda s=s: Y.add_normed_(s[0], s[1], dl.norm1, 0.5, 1e-6) for s in sets]), 0.0, 12 * T * d)
            add("like: RMS norm", timed_graph([lambda s=s: F.rmsnorm(s[1], dl.norm1, 1e-6) for s in sets]), 0.0, 4 * T * d)
            # token input
            sd = c.token_side["dim"]
            ids = torch.randint(0, c.vocab_size, (T,), device=dev, dtype=torch.int32)
            nb = 2 * (2 * sd * d + T * (d + 3 * sd)) + 12 * T * d
            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d)), nb)
            add(f"token input (all kernels), {T} rows", timed_graph([lambda s=s: Y.token_side_(s[0], s[1], ids, dl, model.side_embed, 0.5, 1e-6) for s in sets]),
                4.0 * T * d * sd, nb)
            add("like: its two products as plain GEMMs", timed_graph([lambda s=s: F.gemm(F.gemm(s[1], dl.side_gate), dl.side_proj) for s in sets]), 4.0 * T * d * sd,
                2 * (2 * sd * d + T * (2 * d + 2 * sd)))
            # experts
            ff = next(l.ff for l in model.layers if hasattr(l.ff, "router"))
            mc = ModelConfig(model_type="qwen3_moe", hidden_size=d, num_experts=ff.experts, num_experts_per_tok=ff.top, moe_intermediate_size=ff.ff)
            twin = MoEMLP(mc, bf, dev)
            for prm in twin.parameters():
                prm.normal_(std=0.02)
            used = min(ff.experts, T * ff.top)
            nb = 2 * (3 * used * d * ff.ff + T * ff.top * (2 * d + 2 * ff.ff)) + 12 * T * d
            fl = 6.0 * T * ff.top * d * ff.ff
            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d)), 16 * T * d)
            ms = timed_graph([lambda s=s: Y.feed_forward_(s[0], s[1], ff, dl.norm1, 0.5, 1e-6) for s in sets[:4]])
            add(f"experts with router and join (all kernels), {T} rows", ms, fl, nb)
            ms = timed(lambda: twin(sets[0][1], sets[1][1]), 5, 3) if T > 256 else timed_graph([lambda s=s: twin(s[1], s[1]) for s in sets[:4]])
            add(f"like: Qwen3-MoE block, {T} rows", ms, fl, nb - 8 * T * d)
            del sets, twin
        # attention
        m = at.mixer
        H, G = m.heads, m.kv_heads
        for n, ctx in DECODE:
            b = rows_batch(n, ctx)
            nb = n * ctx * G * (m.dim + m.vdim) * 2
            sets = copies(lambda: (rows(n, m.in_width), *(torch.randn(n * ctx // 64, G, 64, w, device=dev).to(bf) for w in (m.dim, m.vdim))), nb)
            add(f"attention decode (all kernels), {n} x {ctx}", timed_graph([lambda s=s: S.attention(s[0], m, b, s[1], s[2]) for s in sets]), 4.0 * n * ctx * H * m.dim, nb)
            sp = E.choose_splits(n, G, ctx // 2, 64)
            add("like: paged decode attention", timed_graph([lambda s=s: E.paged_decode(s[0][:, : H * m.dim], s[1], s[2], b.block_table, b.seq_lens, H, G, m.dim,
                                                                                      num_splits=sp) for s in sets]), 4.0 * n * ctx * H * m.dim, nb)
            del sets
        for n, length in PREFILL:
            b, T, pairs = portion_batch(n, length), n * length, n * length * length / 2
            kc, vc = (torch.zeros((T // 64, G, 64, w), dtype=bf, device=dev) for w in (m.dim, m.vdim))
            nb = 2 * T * (m.in_width + m.mix_width + G * (m.dim + m.vdim))
            sets = copies(lambda: rows(T, m.in_width), nb)
            add(f"attention prefill (all kernels), {n} x {length}", timed_graph([lambda s=s: S.attention(s, m, b, kc, vc) for s in sets]), 2.0 * pairs * H * (m.dim + m.vdim), nb)
            add("like: flash attention", timed_graph([lambda s=s: F.attention_varlen(s, b.cu_q, length, H, G, m.dim) for s in sets]), 4.0 * pairs * H * m.dim, nb)
            del sets
        # recurrent mixers beside retention at the same heads and state
        class RC:
            rms_norm_eps = 1e-6

        for kind in ("mamba2", "delta"):
            m = pick(kind).mixer
            ret = RetentionMixer(dict(heads=m.heads, dim=m.dim, vdim=m.vdim, rot={"dims": m.dim, "base": 1e4}, decay=[0.99] * m.heads), RC, bf, dev)
            G = m.groups if kind == "mamba2" else m.kv_heads
            for n, _ in DECODE:
                b = rows_batch(n, 64)
                nb = n * m.heads * m.dim * m.vdim * 8
                sets = copies(lambda: (rows(n, m.in_width), torch.randn(n, m.taps, m.channels, device=dev).to(bf), torch.randn(n, m.heads, m.dim, m.vdim, device=dev),
                                       rows(n, ret.in_width)), nb)
                add(f"{kind} decode (all kernels), {n} rows", timed_graph([lambda s=s: S.recurrent(s[0], m, b, s[1], s[2]) for s in sets]), 0.0, nb)
                add("like: retention decode", timed_graph([lambda s=s: X.retention_(s[3], ret, b, s[2]) for s in sets]), 0.0, nb)
                del sets
            for n, length in PREFILL:
                b, T, C = portion_batch(n, length), n * length, X.CHUNK
                ring, st = torch.zeros((n, m.taps, m.channels), dtype=bf, device=dev), torch.zeros((n, m.heads, m.dim, m.vdim), device=dev)
                sets = copies(lambda: (rows(T, m.in_width), rows(T, ret.in_width)), 2 * T * (m.in_width + ret.in_width))
                states = (T // C) * m.heads * m.dim * m.vdim * 16
                nb = 2 * T * (3 * m.channels + 2 * m.heads * m.vdim) + states       # in, convolved, read; gate, out; chunk states
                fl = 2.0 * T * m.heads * (C / 2 * (m.dim + m.vdim) + 2 * m.dim * m.vdim)
                if kind == "delta":      # K K^T, T K, T V, W S more; W, keys, values and writes of the chunks
                    fl += 2.0 * T * m.heads * (C / 2 * (2 * m.dim + m.vdim) + m.dim * m.vdim)
                    nb += 2 * T * m.heads * (4 * m.dim * 2 + 2 * m.vdim * 2 + 2 * m.vdim * 2)
                add(f"{kind} prefill (all kernels), {n} x {length}", timed_graph([lambda s=s: S.recurrent(s[0], m, b, ring, st) for s in sets]), fl, nb)
                nb = 2 * T * m.heads * (3 * m.dim + 3 * m.vdim) + states
                add("like: retention prefill", timed_graph([lambda s=s: X.retention_(s[1], ret, b, st) for s in sets]),
                    2.0 * T * m.heads * (C / 2 * (m.dim + m.vdim) + 2 * m.dim * m.vdim), nb)
                del sets
    return out


def kikivik_table(name: str) -> list:
    """``kernel_table`` of a pre-norm layer-list preset. The like kernels are those of the layer-list models that it is closest to: latent
    attention with an output gate and plain queries, causal grouped attention with biases, clamped experts without a shared unit, normed joins;
    and flash and paged decode attention of the plain models."""
    from rl_b200.models.gated import GatedExperts
    from rl_b200.models.mixers import GroupedAttentionMixer, LatentAttentionMixer
    from rl_b200.ops import layer_ops as Y
    from rl_b200.ops import sequence_ops as S

    pk, c, dev, bf = peaks(), preset(name), "cuda", torch.bfloat16
    model = build_model(c, device=dev, dtype=bf, seed=0)
    la, at = (next(l for l in model.layers if l.mixer.kind == kind) for kind in ("latent_attention", "attention"))
    glu = next(l.ff for l in model.layers if l.ff is not None and not hasattr(l.ff, "router"))
    moe = next(l.ff for l in model.layers if hasattr(l.ff, "router"))
    d, out = c.hidden_size, []

    def add(label, ms, flops=0.0, nbytes=0.0):
        roof = max(flops / pk["flops"], nbytes / pk["hbm"]) * 1e3
        out.append(dict(kernel=label, ms=round(ms, 4), roofline_ms=round(roof, 4), fraction=round(roof / ms, 3)))

    rows = lambda T, n: torch.randn(T, n, device=dev).to(bf)   # noqa: E731
    with torch.no_grad():
        m, g = la.mixer, at.mixer
        for T in (64, 4096):
            # products with what follows them
            for label, w, unit in (("latent in_proj", m.in_proj, None), ("query up-projection", m.q_up, None), ("latent out_proj", m.out_proj, None),
                                   ("attention in_proj", g.in_proj, None), ("gate_up + clamped unit", glu.gate_up, glu), ("gate_up + silu unit", moe.shared.gate_up, moe.shared)):
                N, K = w.shape
                nb = 2 * (N * K + T * (K + (N if unit is None else N // 2)))
                sets = copies(lambda: (rows(T, K), w.detach().clone()), nb)
                fn = Y.linear if unit is None else lambda a, b, unit=unit: Y.gated_linear(a, b, unit.limit)
                add(f"{label} [{N} x {K}], {T} rows", timed_graph([lambda s=s: fn(s[0], s[1]) for s in sets]), 2.0 * T * N * K, nb)
                add("like: plain GEMM", timed_graph([lambda s=s: F.gemm(s[0], s[1]) for s in sets]), 2.0 * T * N * K, 2 * (N * K + T * (N + K)))
                del sets
            # joins, norms, the start
            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d), rows(T, d)), 12 * T * d)
            add(f"join: x += y, next norm, {T} rows", timed_graph([lambda s=s: Y.add_normed_(s[0], s[1], None, 1.0, 1e-6, la.norm1) for s in sets]), 0.0, 12 * T * d)
            add("like: normed join", timed_graph([lambda s=s: Y.add_normed_(s[0], s[1], la.norm1, 0.5, 1e-6) for s in sets]), 0.0, 12 * T * d)
            ids = torch.randint(0, c.vocab_size, (T,), device=dev, dtype=torch.int32)
            add(f"embedding + first norm, {T} rows", timed_graph([lambda: Y.embed(ids, model.embed_tokens, 2.0, la.norm1, 1e-6) for _ in range(8)]), 0.0, 8 * T * d)
            add("like: embedding", timed_graph([lambda: Y.embed(ids, model.embed_tokens, 2.0) for _ in range(8)]), 0.0, 8 * T * d)
            sets = copies(lambda: rows(T, m.in_width), 4 * T * m.q_rank)
            add(f"query latent norm, {T} rows", timed_graph([lambda s=s: Y.group_norm_(s, m.q_norm, 1, 1e-6) for s in sets]), 0.0, 4 * T * m.q_rank)
            add("like: RMS norm", timed_graph([lambda s=s: F.rmsnorm(s[:, : m.q_rank], m.q_norm, 1e-6) for s in sets]), 0.0, 4 * T * m.q_rank)
            del sets
            # experts
            sh = moe.shared
            like = GatedExperts(dict(router={"experts": moe.experts, "top": moe.top, "groups": {"count": 8, "keep": 4}}, expert={"ff": moe.ff, "limit": 7.0}), c, bf, dev)
            for prm in like.parameters():
                prm.normal_(std=0.02)
            used = min(moe.experts, T * moe.top)
            nb = 2 * (3 * used * d * moe.ff + T * moe.top * (2 * d + 2 * moe.ff)) + 12 * T * d
            fl = 6.0 * T * moe.top * d * moe.ff
            nbs, fls = 2 * (3 * d * sh.ff + T * (d + 2 * sh.ff)), 6.0 * T * d * sh.ff
            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d)), 16 * T * d)
            ms = timed_graph([lambda s=s: Y.feed_forward_(s[0], s[1], moe, None, 1.0, 1e-6, la.norm1) for s in sets[:4]])
            add(f"experts with router, shared unit and join (all kernels), {T} rows", ms, fl + fls, nb + nbs)
            ms = timed_graph([lambda s=s: Y.feed_forward_(s[0], s[1], like, la.norm1, 0.5, 1e-6) for s in sets[:4]])
            add("like: clamped experts with router and join", ms, fl, nb)
            del sets, like
        # chunked attention beside causal attention over as many keys as a query sees here
        C = g.chunk
        H, G = g.heads, g.kv_heads
        twin = GroupedAttentionMixer(dict(heads=H, kv_heads=G, dim=g.dim, vdim=g.vdim, scale=g.scale, rot={"dims": g.dim, "base": 1e6}), c, bf, dev)
        for n, ctx in DECODE:
            for label, mx, seen in (("chunked attention", g, ctx - (ctx - 1) // C * C), ("like: causal attention", twin, C)):
                b = rows_batch(n, ctx if mx is g else seen)
                nb, pages = n * seen * G * (g.dim + g.vdim) * 2, n * ctx // 64
                sets = copies(lambda: (rows(n, mx.in_width), *(torch.randn(pages, G, 64, w, device=dev).to(bf) for w in (g.dim, g.vdim)), rows(n, G * g.vdim)), nb)
                add(f"{label} decode (all kernels), {n} rows, {seen} keys seen", timed_graph([lambda s=s: S.attention(s[0], mx, b, s[1], s[2], s[3] if mx.v_mix else None) for s in sets]),
                    4.0 * n * seen * H * g.dim, nb)
                if mx is twin:
                    sp = E.choose_splits(n, G, seen // 2, 64)
                    add("like: paged decode attention", timed_graph([lambda s=s: E.paged_decode(s[0][:, : H * g.dim], s[1], s[2], b.block_table, b.seq_lens, H, G, g.dim, num_splits=sp)
                                                                     for s in sets]), 4.0 * n * seen * H * g.dim, nb)
                del sets
        for n, length in PREFILL:
            for label, mx, per in (("chunked attention", g, min(C, length)), ("like: causal attention", twin, length)):
                b, T = portion_batch(n, length), n * length
                kc, vc = (torch.zeros((T // 64, G, 64, w), dtype=bf, device=dev) for w in (g.dim, g.vdim))
                nb = 2 * T * (mx.in_width + mx.mix_width + G * (g.dim + g.vdim))
                sets = copies(lambda: (rows(T, mx.in_width), rows(T, G * g.vdim)), nb)
                add(f"{label} prefill (all kernels), {n} x {length}", timed_graph([lambda s=s: S.attention(s[0], mx, b, kc, vc, s[1] if mx.v_mix else None) for s in sets]),
                    2.0 * T * per / 2 * H * (g.dim + g.vdim), nb)
                if mx is twin:      # over sequences of a chunk's length
                    cu = torch.arange(0, T + 1, min(C, length), dtype=torch.int32, device=dev)
                    add(f"like: flash attention, {T // min(C, length)} x {min(C, length)}", timed_graph([lambda s=s: F.attention_varlen(s[0], cu, min(C, length), H, G, g.dim) for s in sets]),
                        2.0 * T * min(C, length) / 2 * H * (g.dim + g.vdim), nb)
                del sets
        # latent attention: queries through their latent, no gate, beside gated latent attention whose queries stand in the projected rows
        gated = LatentAttentionMixer(dict(heads=m.heads, dim=m.dim, rot_dim=m.rot_dim, vdim=m.vdim, kv_rank=m.rank, scale=m.scale, rot={"dims": m.rot_dim, "base": 5e5}), c, bf, dev)
        gated.kv_up.normal_(std=0.02)
        qb = m.q_up.numel() * 2
        for n, ctx in DECODE:
            b = rows_batch(n, ctx)
            nb, fl = n * ctx * m.latent_width * 2 + m.kv_up.numel() * 2, 2.0 * n * ctx * m.heads * (2 * m.rank + m.rot_dim)
            sets = copies(lambda: (rows(n, m.in_width), torch.randn(n * ctx // 64, 64, m.latent_width, device=dev).to(bf), rows(n, gated.in_width)), nb)
            add(f"latent attention decode with query up-projection (all kernels), {n} x {ctx}", timed_graph([lambda s=s: X.latent_attention(s[0], m, b, s[1]) for s in sets]), fl, nb + qb)
            add("like: gated latent attention decode", timed_graph([lambda s=s: X.latent_attention_(s[2], gated, b, s[1]) for s in sets]), fl, nb)
            del sets
        for n, length in PREFILL:
            b, T = portion_batch(n, length), n * length
            pairs = n * length * length / 2
            cache = torch.zeros((T // 64, 64, m.latent_width), dtype=bf, device=dev)
            fl = 2.0 * pairs * m.heads * (m.dim + m.rot_dim + m.vdim) + 2.0 * T * m.kv_up.numel()
            nb = 2 * T * (m.in_width + m.q_up.shape[0] + m.mix_width + 2 * m.heads * (m.dim + m.vdim))
            sets = copies(lambda: (rows(T, m.in_width), rows(T, gated.in_width)), nb)
            add(f"latent attention prefill with query up-projection (all kernels), {n} x {length}", timed_graph([lambda s=s: X.latent_attention(s[0], m, b, cache) for s in sets]),
                fl + 2.0 * T * m.q_up.numel(), nb)
            add("like: gated latent attention prefill", timed_graph([lambda s=s: X.latent_attention_(s[1], gated, b, cache) for s in sets]), fl, nb)
            del sets
    return out


def zonidra_table(name: str) -> list:
    """``kernel_table`` of a layer-list preset with norms on both sides. The like kernels are those of Kikivik at the same sizes: its joins, embedding,
    silu experts with a shared unit, chunked soft-max attention; for the polynomial activation the RMS norm over as many columns."""
    from rl_b200.models.gated import GatedExperts
    from rl_b200.models.mixers import GroupedAttentionMixer
    from rl_b200.ops import layer_ops as Y
    from rl_b200.ops import sequence_ops as S

    pk, c, dev, bf = peaks(), preset(name), "cuda", torch.bfloat16
    model = build_model(c, device=dev, dtype=bf, seed=0)
    own, lent = model.layers[0], model.layers[1]
    poly = next(l.ff for l in model.layers if hasattr(l.ff, "coef"))
    moe = next(l.ff for l in model.layers if hasattr(l.ff, "router"))
    d, out = c.hidden_size, []

    def add(label, ms, flops=0.0, nbytes=0.0):
        roof = max(flops / pk["flops"], nbytes / pk["hbm"]) * 1e3
        out.append(dict(kernel=label, ms=round(ms, 4), roofline_ms=round(roof, 4), fraction=round(roof / ms, 3)))

    rows = lambda T, n: torch.randn(T, n, device=dev).to(bf)   # noqa: E731
    with torch.no_grad():
        g = own.mixer
        for T in (64, 4096):
            for label, w in (("in_proj", g.in_proj), ("in_proj without keys and values", lent.mixer.in_proj), ("out_proj", g.out_proj), ("up", poly.up), ("down", poly.down),
                             ("router and shared gate", moe.router)):
                N, K = w.shape
                nb = 2 * (N * K + T * (K + N)) + (2 * T * N if w is moe.router else 0)
                sets = copies(lambda: (rows(T, K), w.detach().clone()), nb)
                fn = Y.router_logits if w is moe.router else Y.linear
                add(f"{label} [{N} x {K}], {T} rows", timed_graph([lambda s=s: fn(s[0], s[1]) for s in sets]), 2.0 * T * N * K, nb)
                add("like: plain GEMM", timed_graph([lambda s=s: F.gemm(s[0], s[1]) for s in sets]), 2.0 * T * N * K, 2 * (N * K + T * (N + K)))
                del sets
            sets = copies(lambda: rows(T, poly.ff), 4 * T * poly.ff)
            one = torch.ones(poly.ff, dtype=bf, device=dev)
            add(f"polynomial activation, {T} rows", timed_graph([lambda s=s: Y.poly_norm_(s, poly.coef, poly.ff, 1e-6) for s in sets]), 0.0, 4 * T * poly.ff)
            add("like: RMS norm", timed_graph([lambda s=s: F.rmsnorm(s, one, 1e-6) for s in sets]), 0.0, 4 * T * poly.ff)
            del sets
            # joins: T single rows, and one portion of T rows
            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d)), 12 * T * d)
            add(f"join: x += ls norm(y), next norm, {T} rows", timed_graph([lambda s=s: Y.join(s[0], s[1], own.norm1b, 1.0, 1e-6, own.norm2, ls=own.ls1) for s in sets]), 0.0, 12 * T * d)
            add("like: join and next norm", timed_graph([lambda s=s: Y.join(s[0], s[1], None, 1.0, 1e-6, own.norm2) for s in sets]), 0.0, 12 * T * d)
            b = rows_batch(T, 64) if T == 64 else portion_batch(1, T)
            b.state_rows = b.state_rows + 1
            b.row_state = b.row_state + 1 if b.row_state is not None else None
            carry = Y.Carry(T + 1 if T == 64 else 2, 2, d, True, dev)
            state = 8 * T * d if T == 64 else 0
            sh = Y.Shift(own.shift, 0, carry, b)
            add(f"join with token shift, {T} rows", timed_graph([lambda s=s: Y.join(s[0], s[1], own.norm1b, 1.0, 1e-6, own.norm1, ls=own.ls1, shift=sh) for s in sets]), 0.0, 12 * T * d + state)
            add("like: join and next norm", timed_graph([lambda s=s: Y.join(s[0], s[1], None, 1.0, 1e-6, own.norm1) for s in sets]), 0.0, 12 * T * d)
            del sets
            b.ids = torch.randint(0, c.vocab_size, (T,), device=dev, dtype=torch.int32)
            add(f"embedding with pairs, first norm, token shift, {T} rows", timed_graph([lambda: Y.start(b, model.embed_tokens, 2.0, own.norm1, 1e-6, model.bigram, c.bigram, sh) for _ in range(8)]), 0.0,
                10 * T * d + state)
            add("like: embedding + first norm", timed_graph([lambda: Y.embed(b.ids, model.embed_tokens, 2.0, own.norm1, 1e-6) for _ in range(8)]), 0.0, 8 * T * d)
            # experts
            unit = moe.shared
            like = GatedExperts(dict(router={"experts": moe.experts, "top": moe.top}, expert={"ff": moe.ff}, shared={"ff": unit.ff}, weigh_input=True, corrected=False), c, bf, dev)
            for prm in like.parameters():
                prm.normal_(std=0.02)
            nbs, fls = 2 * (3 * d * unit.ff + T * (d + 2 * unit.ff)), 6.0 * T * d * unit.ff

            def cost(copies_):
                used = min(moe.experts, copies_)
                return 6.0 * copies_ * d * moe.ff + fls, 2 * (3 * used * d * moe.ff + copies_ * (2 * d + 2 * moe.ff)) + 12 * T * d + nbs

            sets = copies(lambda: (torch.randn(T, d, device=dev), rows(T, d)), 16 * T * d)
            real = round(T * moe.top * moe.experts / moe.outputs)
            ms = timed_graph([lambda s=s: Y.feed_forward(s[0], s[1], moe, own.norm1b, 1.0, 1e-6, own.norm1, own.ls1) for s in sets[:4]])
            add(f"experts with identity outputs, router, gated shared unit and join (all kernels), {T} rows", ms, *cost(real))
            ms = timed_graph([lambda s=s: Y.feed_forward(s[0], s[1], like, None, 1.0, 1e-6, own.norm1) for s in sets[:4]])
            add("like: experts with router, shared unit and join", ms, *cost(T * moe.top))
            del sets, like
        # attention beside chunked soft-max attention over as many keys as a query sees here
        W, H, G = g.window, g.heads, g.kv_heads
        twin = GroupedAttentionMixer(dict(heads=H, kv_heads=G, dim=g.dim, vdim=g.vdim, scale=g.scale, rot={"dims": g.dim, "base": 1e6}, bias=False, interleaved=False), c, bf, dev)
        m2 = lent.mixer
        for n, ctx in DECODE:
            seen = min(ctx, W) + g.keep
            for label, mx, keys in (("windowed sigmoid attention", g, seen), ("the same on another layer's keys", m2, seen), ("like: soft-max attention", twin, -(-seen // 64) * 64)):
                b, pages = rows_batch(n, ctx if mx is not twin else keys), n * ctx // 64
                nb = n * keys * G * (g.dim + g.vdim) * 2
                sets = copies(lambda: (rows(n, mx.in_width), *(torch.randn(pages, G, 64, w, device=dev).to(bf) for w in (g.dim, g.vdim))), nb)
                add(f"{label} decode (all kernels), {n} rows, {keys} keys seen", timed_graph([lambda s=s: S.attention(s[0], mx, b, s[1], s[2]) for s in sets]), 4.0 * n * keys * H * g.dim, nb)
                del sets
        for n, length in PREFILL:
            for label, mx in (("windowed sigmoid attention", g), ("like: soft-max attention", twin)):
                b, T = portion_batch(n, length), n * length
                size = min(W, length) if mx is g else length
                pairs = n * (size * (size + 1) / 2 + (length - size) * size)
                if mx is g:
                    pairs += n * g.keep * max(0, length - size)
                kc, vc = (torch.zeros((T // 64, G, 64, w), dtype=bf, device=dev) for w in (g.dim, g.vdim))
                nb = 2 * T * (mx.in_width + mx.mix_width + G * (g.dim + g.vdim))
                sets = copies(lambda: rows(T, mx.in_width), nb)
                add(f"{label} prefill (all kernels), {n} x {length}", timed_graph([lambda s=s: S.attention(s, mx, b, kc, vc) for s in sets]), 2.0 * pairs * H * (g.dim + g.vdim), nb)
                del sets
    return out


def zonidra_main(steps: int = 5, warmup: int = 3, sizes=None, clocks=None) -> int:
    torch.backends.cuda.matmul.allow_tf32 = False
    L.lib()
    res = dict(metric="layer-list model with norms on both sides, serving (device time)", unit="tokens/s", dtype="bf16", data="synthetic (random weights and tokens)", models={}, kernels={})
    for name in sizes or ZONIDRA:
        for kind in ("zonidra", "kikivik"):
            res["models"][f"{name}:{kind}"] = serving_row(preset(name) if kind == "zonidra" else kikivik_twin(name), steps, warmup)
        res["kernels"][name] = zonidra_table(name)
        torch.cuda.empty_cache()
    return finish(res, clocks)


def kikivik_main(steps: int = 5, warmup: int = 3, sizes=None, clocks=None) -> int:
    torch.backends.cuda.matmul.allow_tf32 = False
    L.lib()
    res = dict(metric="pre-norm layer-list model serving (device time)", unit="tokens/s", dtype="bf16", data="synthetic (random weights and tokens)", models={}, kernels={})
    for name in sizes or KIKIVIK:
        for kind in ("kikivik", "qwen3_moe"):
            res["models"][f"{name}:{kind}"] = serving_row(preset(name) if kind == "kikivik" else moe_twin(name), steps, warmup)
        res["kernels"][name] = kikivik_table(name)
        torch.cuda.empty_cache()
    return finish(res, clocks)


def redarax_main(steps: int = 5, warmup: int = 3, sizes=None, clocks=None) -> int:
    torch.backends.cuda.matmul.allow_tf32 = False
    L.lib()
    res = dict(metric="post-norm layer-list model serving (device time)", unit="tokens/s", dtype="bf16", data="synthetic (random weights and tokens)", models={}, kernels={})
    for name in sizes or REDARAX:
        for kind in ("redarax", "qwen3_moe"):
            res["models"][f"{name}:{kind}"] = serving_row(preset(name) if kind == "redarax" else moe_twin(name), steps, warmup)
        res["kernels"][name] = redarax_table(name)
        torch.cuda.empty_cache()
    return finish(res, clocks)


def serving_row(cfg: ModelConfig, steps: int, warmup: int) -> dict:
    row = dict(weights_gb=round(2e-9 * cfg.num_parameters(), 2), runs=len(cfg.layer_runs))
    need = max(max(n * c for n, c in DECODE), max(n * c for n, c in PREFILL))
    eng = engine_for(cfg, need, max(n for n, _ in DECODE), max(c for _, c in DECODE) + 64)
    for n, length in PREFILL:
        ms = prefill_ms(eng, n, length, steps, warmup)
        row[f"prefill {n}x{length}"] = dict(ms=round(ms, 3), tokens_per_s=round(n * length / ms * 1e3))
    for n, ctx in DECODE:
        ms = decode_ms(eng, n, ctx, steps, warmup)
        row[f"decode {n}x{ctx}"] = dict(ms=round(ms, 3), tokens_per_s=round(n / ms * 1e3))
    eng.sleep(True)
    del eng
    torch.cuda.empty_cache()
    return row


def finish(res: dict, clocks) -> int:
    res["status"] = L.check_status()
    if clocks is not None:
        res["clocks"] = clocks()
    print(json.dumps(res), flush=True)
    return 0


def main(steps: int = 5, warmup: int = 3, sizes=None, clocks=None) -> int:
    torch.backends.cuda.matmul.allow_tf32 = False
    L.lib()
    res = dict(metric="layer-list model serving (device time)", unit="tokens/s", dtype="bf16", data="synthetic (random weights and tokens)", models={}, kernels={})
    for name in sizes or SIZES:
        for kind in ("gadarax", "llama"):
            res["models"][f"{name}:{kind}"] = serving_row(preset(name) if kind == "gadarax" else llama_twin(name), steps, warmup)
        res["kernels"][name] = kernel_table(name)
        torch.cuda.empty_cache()
    return finish(res, clocks)
