"""Redarax (post-norm layer-list models) on the GPU: the native kernels of both precisions against the float64 oracle, the tensor-core and
single-step forms against the plain kernels at many shapes, and generation through captured decode steps."""

import math

import pytest
import redarax_cases as R
import redarax_oracle as O
import torch
from test_redarax import Cfg, standout_case

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import preset
from rl_b200.models.mixers import DeltaMixer, GroupedAttentionMixer, Mamba2LayerMixer
from rl_b200.models.gated import GatedExperts, GatedUnit
from rl_b200.models.transformer import build_model
from rl_b200.ops import layer_ops as Y
from rl_b200.ops import lib as L
from rl_b200.ops import mixer_ops as X
from rl_b200.ops import sequence_ops as S

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
# sizes that every tensor-core kernel takes, wide enough for the weight-streaming product
TILED = R.config([(R.delta(heads=4, kv_heads=2, dim=40, vdim=72, conv=4), R.dense(ff=136)), (R.attention(heads=6, kv_heads=2, dim=48, vdim=40, rot_dims=32, scale=0.2), R.moe(experts=16, top=3, ff=40, groups=(4, 2))),
                  (R.mamba2(heads=6, vdim=24, state=56, groups=2, norm_groups=3, conv=3), None), (R.attention(heads=4, kv_heads=1, dim=128, vdim=128, rot_dims=128, scale=0.1), R.dense(ff=72)),
                  (R.delta(heads=2, kv_heads=2, dim=128, vdim=128, conv=2), R.moe(experts=8, top=2, ff=64, groups=None))], width=264, vocab=200, side=24)
CASES = dict(R.CASES, tiled=TILED)


@pytest.fixture(autouse=True)
def _clean(native_lib):
    yield
    assert L.check_status() == 0


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request, tmp_path_factory):
    cfg = CASES[request.param]
    w = R.weights(cfg, seed=7)
    path = tmp_path_factory.mktemp(request.param)
    return cfg, w, {dt: R.load(cfg, w, path, DEV, dt) for dt in (F32, BF)}


def rel(a, b):
    return ((a.float() - b.float()).norm() / b.float().norm()).item()


def gaps(got, want):
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / s.pow(2).mean().sqrt()


def close(cfg, w, toks, got, dt):
    """fp32: every position. bf16: the median, and every position up to the first one where a router's choice is within a rounding."""
    g = gaps(got, R.oracle(cfg, w, toks))
    if dt == F32:
        return g.max() < 5e-4
    flip = R.close_routes(cfg, w, toks, 0.05).nonzero()
    n = int(flip[0]) if len(flip) else len(toks)
    return g.median() < 0.08 and (n == 0 or g[:n].max() < 0.3)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [17, 2, 33, 1], [130, 1]])
def test_portions_equal_the_oracle(case, dt, cuts):
    cfg, w, models = case
    toks = R.tokens(cfg, 90 if cuts == [1] else 200)
    eng = R.engine(models[dt], block_size=64, pages=6)
    assert close(cfg, w, toks, R.run_cut(eng, "a", toks, cuts), dt)


@pytest.mark.parametrize("dt", [F32, BF])
def test_mixed_batches_and_reused_pages(case, dt):
    cfg, w, models = case
    seqs = {f"r{i}": R.tokens(cfg, n, seed=i) for i, n in enumerate([150, 1, 33, 17, 90, 2, 160, 16])}
    steps = R.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = R.engine(models[dt], pages=R.live_pages(steps, 32), block_size=32)
    got = R.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert close(cfg, w, t, got[r], dt), r
    assert eng.sched.num_free_blocks == eng.num_blocks


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation(case, graphs):
    """fp32: the tokens the oracle picks, through the scheduler, chunked prefill and (captured) multi-step decode windows."""
    cfg, w, models = case
    prompts = [R.tokens(cfg, n, seed=n) for n in (1, 5, 64, 65, 40, 5)]
    prompts[5] = list(prompts[1])
    eng = R.engine(models[F32], pages=20, block_size=64, requests=3, max_prefill_tokens=48, use_cuda_graphs=graphs)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=20))
    for p, r in zip(prompts, recs):
        z = R.oracle(cfg, w, p + r.out_tokens)[len(p) - 1 : -1]
        top = z.topk(2, -1)
        clear = top[0][:, 0] - top[0][:, 1] > 1e-2
        assert (top[1][:, 0] == torch.tensor(r.out_tokens))[clear].all()
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert torch.allclose(lp, torch.tensor(r.out_logprobs, dtype=F64), atol=5e-3)
    assert bool(eng._graphs) == graphs


def test_long_decoding_keeps_to_the_prefill(case):
    """300 decoded tokens (captured steps, windows, page borders): the log-probabilities are those of one prefill of the same tokens."""
    cfg, w, models = case
    eng = R.engine(models[BF], pages=14, block_size=64, requests=2, use_cuda_graphs=True)
    recs = eng.generate([R.tokens(cfg, 3, 1), R.tokens(cfg, 70, 2)], SamplingParams(temperature=1.0, max_new_tokens=300, seed=3))
    eng.sleep(False)
    for r in recs:
        z = R.run_cut(eng, "x", r.prompt + r.out_tokens, [1000])[len(r.prompt) - 1 : -1]
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert (lp - torch.tensor(r.out_logprobs)).abs().median() < 0.1


@pytest.mark.parametrize("shape", [dict(heads=4, kv_heads=2, dim=16, vdim=24), dict(heads=6, kv_heads=2, dim=128, vdim=128), dict(heads=3, kv_heads=3, dim=7, vdim=5)])
@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 127, 128, 191, 255])
@pytest.mark.parametrize("n", [1, 3, 40, 256])
def test_one_key_far_away(shape, far, n, dt):
    T, bs = 256, 64
    m, p, b, kc, vc, want = standout_case(T, bs, far, n, DEV, dt, **shape)
    with torch.no_grad():
        got = S.attention(p, m, b, kc, vc)[:, : m.heads * m.vdim].float().cpu()
    rows = [i for i in range(n) if T - n + i >= far]
    assert rel(got[rows], want[rows]) < (1e-3 if dt == F32 else 8e-3)
    hidden = [i for i in range(n) if T - n + i < far]
    assert not hidden or rel(got[hidden], want[hidden]) > 0.3


# ------------------------------------------------------------------------------------------------ tensor-core forms against the plain kernels
def batch(lens, starts, bs=64, tiles=True):
    order = sorted(range(len(lens)), key=lambda j: lens[j])
    new, pos0 = [lens[j] for j in order], [starts[j] for j in order]
    pos = torch.cat([torch.arange(s, s + n) for s, n in zip(pos0, new)]).int()
    pages = [-(-(s + n) // bs) for s, n in zip(pos0, new)]
    free = torch.randperm(sum(pages) + 3).tolist()
    own = [[free.pop() for _ in range(n)] for n in pages]
    slot = lambda k, lo: torch.tensor([own[k][t // bs] * bs + t % bs for t in range(lo, pos0[k] + new[k])])  # noqa: E731
    bt = torch.zeros(len(new), max(pages) + 1, dtype=torch.int32)
    for k, o in enumerate(own):
        bt[k, : len(o)] = torch.tensor(o)
    of = torch.repeat_interleave(torch.arange(len(new)), torch.tensor(new))
    tl = [k for k, n in enumerate(new) if n > X.PAGED_PORTION] if tiles else []
    n_paged, ns = sum(new[: tl[0]]) if tl else len(pos), sum(n == 1 for n in new)
    srow = torch.randperm(len(new) + 3)[: len(new)]
    b = X.TokenBatch(ids=None, positions=pos.to(DEV), slots=torch.cat([slot(k, pos0[k]) for k in range(len(new))]).to(DEV), n_single=ns, n_paged=n_paged,
                     block_table=bt[of[:n_paged]].to(DEV), seq_lens=(pos[:n_paged] + 1).to(DEV), max_ctx=int(pos.max()) + 1,
                     state_rows=srow.to(DEV), row_state=srow[of].to(DEV), row_off=torch.cat([torch.arange(n) for n in new]).int().to(DEV))
    if ns < len(new):
        b.cu = torch.tensor([0] + torch.tensor(new[ns:]).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
        b.piece_chunk, b.chunk_row, b.chunk_rows = (t.to(DEV) for t in X.chunk_lists(new[ns:]))
    if tl:
        cu = torch.zeros(2, len(tl) + 1, dtype=torch.int32)
        cu[0, 1:] = torch.tensor([new[k] for k in tl]).cumsum(0)
        cu[1, 1:] = torch.tensor([pos0[k] + new[k] for k in tl]).cumsum(0)
        b.cu_q, b.cu_ctx = cu.to(DEV)
        b.whole = all(pos0[k] == 0 for k in tl)
        b.q_tiles, b.ctx_slots = sum(-(-new[k] // 128) for k in tl), torch.cat([slot(k, 0) for k in tl]).to(DEV)
    return b, sum(pages) + 3


@pytest.mark.parametrize("shape", [(6, 2, 48, 40, 32, [1, 77, 5, 100, 17], [299, 0, 0, 29, 623]), (16, 4, 128, 128, 64, [1, 200, 128, 2, 1], [999, 0, 0, 127, 0]),
                                   (8, 1, 64, 96, 64, [300, 33], [0, 0]), (2, 2, 16, 256, 0, [300, 20, 1], [0, 480, 69]), (9, 3, 256, 8, 200, [70, 1], [3, 64])])
def test_attention_kernels(shape):
    H, G, dim, vdim, rd, lens, starts = shape
    torch.manual_seed(0)
    m = GroupedAttentionMixer(R.attention(heads=H, kv_heads=G, dim=dim, vdim=vdim, rot_dims=rd, scale=1.5 / math.sqrt(dim))["mixer"], Cfg, BF, DEV)
    with torch.no_grad():
        m.q_norm.uniform_(0.5, 1.5), m.k_norm.uniform_(0.5, 1.5)
    out = []
    for tiles in (False, True):
        torch.manual_seed(1)
        b, pages = batch(lens, starts, tiles=tiles)
        kc, vc = torch.randn(pages, G, 64, dim, device=DEV).to(BF), torch.randn(pages, G, 64, vdim, device=DEV).to(BF)
        p = torch.randn(b.rows, m.in_width + 16, device=DEV).to(BF)
        keep = S.decode_tiles
        try:
            if not tiles:
                S.decode_tiles = lambda *a: False
            with torch.no_grad():
                y = S.attention(p, m, b, kc, vc)[:, : H * vdim]
        finally:
            S.decode_tiles = keep
        out.append((y, kc, vc))
    assert S.portion_tiles(m, BF) and rel(out[1][0], out[0][0]) < 6e-3
    assert torch.equal(out[0][1], out[1][1]) and torch.equal(out[0][2], out[1][2])


REC = [R.mamba2(heads=6, vdim=24, state=56, groups=2, norm_groups=3, conv=3), R.mamba2(heads=4, vdim=128, state=128, groups=1, norm_groups=1, conv=4),
       R.mamba2(heads=3, vdim=200, state=264, groups=3, norm_groups=1, conv=5), R.mamba2(heads=8, vdim=8, state=8, groups=4, norm_groups=2, conv=2),
       R.delta(heads=4, kv_heads=2, dim=40, vdim=72, conv=4), R.delta(heads=6, kv_heads=2, dim=128, vdim=128, conv=4), R.delta(heads=2, kv_heads=1, dim=8, vdim=8, conv=1),
       R.delta(heads=3, kv_heads=3, dim=64, vdim=120, conv=3), R.delta(heads=4, kv_heads=4, dim=104, vdim=64, conv=6)]


@pytest.mark.parametrize("slow", [False, True])
@pytest.mark.parametrize("lens,starts", [([1, 2, 100, 300, 128, 1], [5, 0, 77, 0, 128, 0]), ([1, 129, 1000], [0, 0, 300]), ([260, 64, 3], [0, 64, 4])])
@pytest.mark.parametrize("entry", REC)
def test_recurrent_kernels(entry, lens, starts, slow):
    """Chunked and single-step kernels against the token-by-token kernel: the states agree to fp32 rounding. ``slow``: decays near 1, beta near 1
    and keys that repeat, so that the writes of a chunk depend on one another."""
    torch.manual_seed(1)
    m = (DeltaMixer if entry["type"] == "delta" else Mamba2LayerMixer)(entry["mixer"], Cfg, BF, DEV)
    b, _ = batch(lens, starts)
    n = len(lens) + 3
    with torch.no_grad():
        m.conv.normal_(std=0.6)
        m.A_log.normal_(mean=-3.0 if slow else 0.0), m.dt_bias.normal_(mean=-2.0), m.norm.uniform_(0.5, 1.5)
        if entry["type"] == "mamba2":
            m.conv_bias.normal_(std=0.3), m.D.normal_()
    p = torch.randn(b.rows, m.in_width + 40, device=DEV)
    if slow and entry["type"] == "delta":
        p[:, m.b_off : m.b_off + m.heads] += 3.0
        p[:, : 2 * m.kv_heads * m.dim] *= 0.3
        p[:, : 2 * m.kv_heads * m.dim] += 1.0
    p = p.to(BF)
    ring, state = torch.randn(n, m.taps, m.channels, device=DEV).to(BF), torch.randn(n, m.heads, m.dim, m.vdim, device=DEV)
    out = []
    for plain in (True, False):
        r, s = ring.clone(), state.clone()
        with torch.no_grad():
            out.append((S.recurrent(p.clone(), m, b, r, s, plain=plain)[:, : m.heads * m.vdim], s, r))
    (want, Sw, rw), (got, Sg, rg) = out
    assert S.rec_tiles(p, m)
    assert rel(got, want) < 3e-3 and (Sg - Sw).abs().max() < 3e-4 * Sw.abs().max()
    live = set(b.state_rows.tolist())
    for j in range(n):
        if j not in live:
            assert torch.equal(Sg[j], state[j]) and torch.equal(rg[j], ring[j])
    ends = {int(r): int(b.positions[e - 1]) for r, (s, e) in zip(b.state_rows.tolist(), S._pieces(b))}
    for r, last in ends.items():      # what a later token will read
        for t in range(max(0, last - m.taps + 2), last + 1):
            assert torch.equal(rg[r, t % m.taps], rw[r, t % m.taps])


@pytest.mark.parametrize("T", [1, 40, 300, 1500])
@pytest.mark.parametrize("spec,width", [(R.moe(experts=16, top=3, ff=40, groups=(4, 2)), 264), (R.moe(experts=64, top=8, ff=64, groups=(8, 4)), 256),
                                        (R.moe(experts=5, top=2, ff=7, groups=None), 61), (R.moe(experts=8, top=8, ff=24, groups=(1, 1)), 64)])
def test_expert_kernels(spec, width, T):
    """Routing, placement, grouped products and the combining join of bf16 rows beside the module's statement; fp32 beside float64."""
    class C2(Cfg):
        hidden_size = width
    torch.manual_seed(0)
    w = {k: v.to(F64) for k, v in O.below(R.weights(R.config([(R.delta(), spec)], width=width), 5), "l0.mlp.").items()}
    h = torch.randn(T, width, dtype=F64).to(BF)
    nw = torch.rand(width) + 0.5
    for dt, tol in ((F32, 1e-4), (BF, 0.02)):
        m = R.module_weights(GatedExperts(spec, C2, dt, DEV), w)
        x = torch.zeros(T, width, device=DEV)
        with torch.no_grad():
            z = Y.router_logits(h.to(DEV, dt), m.router)
            assert torch.allclose(z.double().cpu(), h.double() @ w["router"].T, atol=1e-4)
            Y.feed_forward_(x, h.to(DEV, dt), m, nw.to(DEV, dt), 0.7, 1e-3)
        ref = GatedExperts(spec, C2, F32, "cpu")
        R.module_weights(ref, w)
        with torch.no_grad():
            y = ref(h.float()).double()
        want = 0.7 * O.rms(y, 1e-3) * nw.to(dt).double()
        bad = ((x.double().cpu() - want).norm(dim=-1) / want.norm(dim=-1)) > tol      # (rows with a tie within rounding aside)
        assert bad.sum() <= (0 if dt == F32 else max(1, T // 100))
    assert all(int(c.abs().sum()) == 0 for c in Y._COUNTS.values())


@pytest.mark.parametrize("M,N,K", [(1, 64, 64), (5, 400, 328), (64, 2048, 4096), (300, 1104, 320), (257, 96, 72), (130, 38, 61), (3, 200, 520)])
@pytest.mark.parametrize("dt", [F32, BF])
def test_products(M, N, K, dt):
    """All three product kernels with bias, clamped unit, gated token input and soft cap, beside an fp32 statement."""
    torch.manual_seed(0)
    a, w, bias = torch.randn(M, K, device=DEV).to(dt), (torch.randn(N, K, device=DEV) * 1.5 / math.sqrt(K)).to(dt), torch.randn(N, device=DEV).to(dt)
    tol = 1e-5 if dt == F32 else 5e-3
    ref = (a.double() @ w.double().T).float()
    assert rel(Y.linear(a, w, bias), ref + bias.float()) < tol
    assert rel(Y.linear(a, w, glu=1.3), Y.clamped_glu_ref(ref.cpu(), 1.3).to(DEV)) < tol
    assert rel(Y.capped_logits(a, w, 3.0, 4.0), 4 * torch.tanh(ref * 3 / 4)) < 1e-4
    assert rel(Y.capped_logits(a, w, 3.0, 0.0), ref * 3) < 1e-4

    class Layer:
        side_dim, layer_idx, side_gate, side_proj, side_norm = N - 3, 2, w, torch.randn(40, N, device=DEV).to(dt), torch.ones(40, device=DEV).to(dt)
    table = torch.randn(50, 3 * Layer.side_dim, device=DEV).to(dt)
    ids = torch.randint(0, 50, (M,), device=DEV, dtype=torch.int32)
    x = torch.zeros(M, 40, device=DEV)
    Y.token_side_(x, a, ids, Layer, table, 1.0, 1e-6)
    g = torch.nn.functional.gelu(ref[:, : N - 3], approximate="tanh") * table[ids.long(), 2 * Layer.side_dim :].float()
    y = g.to(dt).float() @ Layer.side_proj[:, : N - 3].float().T
    assert rel(x, y * torch.rsqrt(y.pow(2).mean(-1, keepdim=True) + 1e-6)) < 2 * tol


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("d", [37, 264, 2048, 4096, 9000])
def test_joins(d, dt):
    torch.manual_seed(0)
    for rows in (3, 700):
        x, y, w, nw = torch.randn(rows, d, device=DEV), torch.randn(rows, d, device=DEV).to(dt), torch.randn(d, device=DEV).to(dt), torch.randn(d, device=DEV).to(dt)
        want = x.double() + 0.7 * O.rms(y.double(), 1e-3) * w.double()
        for norm in (None, nw):
            x1 = x.clone()
            h = Y.add_normed_(x1, y, w, 0.7, 1e-3, norm)
            assert rel(x1, want) < 1e-6 and rel(h, want if norm is None else O.rms(want, 1e-3) * nw.double()) < (1e-6 if dt == F32 else 4e-3)
        if d % 3 == 0:
            z = y.clone()
            Y.group_norm_(z, w, 3, 1e-3)
            assert rel(z, O.rms(y.double().view(rows, 3, -1), 1e-3).view(rows, d) * w.double()) < (1e-6 if dt == F32 else 4e-3)


def test_dense_unit_of_odd_width():
    m = R.module_weights(GatedUnit(R.dense(ff=13), Cfg, BF, DEV), {k: v for k, v in O.below(R.weights(R.config([(R.delta(), R.dense(ff=13))]), 1), "l0.mlp.").items()})
    h = torch.randn(70, 56, device=DEV).to(BF)
    with torch.no_grad():
        assert rel(Y.linear(Y.linear(h, m.gate_up, glu=m.limit), m.down), m(h)) < 1e-2


def test_presets_generate_with_captured_steps():
    m = build_model(preset("tiny-redarax"), device=DEV, dtype=BF, seed=1)
    prompts = [R.tokens({"vocab": 264}, n, n) for n in (5, 70, 129, 1)]
    outs = []
    for graphs in (True, False):
        eng = R.engine(m, pages=40, block_size=64, use_cuda_graphs=graphs)
        outs.append([r.out_tokens for r in eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))])
        assert bool(eng._graphs) == graphs
    assert outs[0] == outs[1]
