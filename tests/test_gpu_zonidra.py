"""Zonidra on the GPU: the native kernels of both precisions against the float64 oracle, the tensor-core forms against the plain kernels at many
shapes, and generation through captured decode steps."""

import math

import pytest
import torch
import zonidra_cases as Z
import zonidra_oracle as O
from test_gpu_redarax import batch
from test_zonidra import Cfg, build, pieces, unit
from test_zonidra import test_start_and_shift_over_steps as start_and_shift

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import preset
from rl_b200.models.transformer import build_model
from rl_b200.ops import layer_ops as Y
from rl_b200.ops import lib as L
from rl_b200.ops import mixer_ops as X
from rl_b200.ops import sequence_ops as S

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
# sizes that every tensor-core kernel takes, wide enough for the weight-streaming product; windows across and inside tiles of 64 and 128 keys
TILED = Z.config([(Z.attention(heads=6, kv_heads=2, dim=48, vdim=128, rot_dims=32, scale=0.2, size=100, keep=70), Z.moe(experts=14, identity=2, top=3, ff=40, shared=72)),
                  (Z.attention(heads=4, kv_heads=2, dim=128, vdim=128, rot_dims=128, scale=0.1, size=33, keep=5), Z.dense(ff=136)),
                  (Z.attention(heads=8, kv_heads=2, dim=128, vdim=128, rot_dims=64, scale=0.1, size=70, keep=0, source=1), None),
                  (Z.attention(heads=2, kv_heads=2, dim=48, vdim=128, rot_dims=20, scaling=None, scale=0.2, size=0, source=0), Z.dense(ff=72)),
                  (Z.attention(heads=8, kv_heads=1, dim=128, vdim=128, rot_dims=128, scale=0.1, size=64, keep=130), Z.moe(experts=8, identity=0, top=2, ff=64, shared=0))], width=264, vocab=200)
CASES = dict(Z.CASES, tiled=TILED)


@pytest.fixture(autouse=True)
def _clean(native_lib):
    yield
    assert L.check_status() == 0


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request, tmp_path_factory):
    cfg = CASES[request.param]
    w = Z.weights(cfg, seed=7)
    path = tmp_path_factory.mktemp(request.param)
    return cfg, w, {dt: Z.load(cfg, w, path, DEV, dt) for dt in (F32, BF)}


def rel(a, b):
    return ((a.double().cpu() - b.double().cpu()).norm() / b.double().cpu().norm()).item()


def gaps(got, want):
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / s.pow(2).mean().sqrt()


_SEEN: dict = {}


def oracle(cfg, w, toks, margin=None):
    """The oracle's logits (with ``margin`` the positions of close routes), computed once per sequence."""
    key = (id(w), tuple(toks), margin)
    if key not in _SEEN:
        _SEEN[key] = Z.oracle(cfg, w, toks) if margin is None else Z.close_routes(cfg, w, toks, margin)
    return _SEEN[key]


def close(cfg, w, toks, got, dt):
    """fp32: every position. bf16: the median, and every position up to the first one where a router's choice is within a rounding."""
    g = gaps(got, oracle(cfg, w, toks))
    if dt == F32:
        return g.max() < 5e-4
    flip = oracle(cfg, w, toks, 0.03).nonzero()
    n = int(flip[0]) if len(flip) else len(toks)
    return g.median() < 0.08 and (n == 0 or g[:n].max() < 0.3)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [17, 2, 33, 1], [130, 1], [100, 70, 1]])
def test_portions_equal_the_oracle(case, dt, cuts):
    cfg, w, models = case
    toks = Z.tokens(cfg, 90 if cuts == [1] else 300)
    eng = Z.engine(models[dt], block_size=64, pages=6)
    assert close(cfg, w, toks, Z.run_cut(eng, "a", toks, cuts), dt)


@pytest.mark.parametrize("dt", [F32, BF])
def test_mixed_batches_and_reused_pages(case, dt):
    cfg, w, models = case
    seqs = {f"r{i}": Z.tokens(cfg, n, seed=i) for i, n in enumerate([150, 1, 33, 17, 90, 2, 160, 16])}
    steps = Z.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = Z.engine(models[dt], pages=Z.live_pages(steps, 32), block_size=32)
    got = Z.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert close(cfg, w, t, got[r], dt), r
    assert eng.sched.num_free_blocks == eng.num_blocks


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation(case, graphs):
    """fp32: the tokens the oracle picks, through the scheduler, portions and (captured) multi-step decode windows."""
    cfg, w, models = case
    prompts = [Z.tokens(cfg, n, seed=n) for n in (1, 5, 64, 65, 140, 5)]
    prompts[5] = list(prompts[1])
    prompts.append(prompts[4][:129])
    eng = Z.engine(models[F32], pages=20, block_size=64, requests=3, max_prefill_tokens=48, use_cuda_graphs=graphs)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=20))
    for p, r in zip(prompts, recs):
        z = oracle(cfg, w, p + r.out_tokens)[len(p) - 1 : -1]
        top = z.topk(2, -1)
        clear = top[0][:, 0] - top[0][:, 1] > 1e-2
        assert (top[1][:, 0] == torch.tensor(r.out_tokens))[clear].all()
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert torch.allclose(lp, torch.tensor(r.out_logprobs, dtype=F64), atol=5e-3)
    assert bool(eng._graphs) == graphs


def test_long_decoding_keeps_to_the_prefill(case):
    """300 decoded tokens (captured steps, windows, page borders): the log-probabilities are those of one prefill of the same tokens."""
    cfg, w, models = case
    eng = Z.engine(models[BF], pages=14, block_size=64, requests=2, use_cuda_graphs=True)
    recs = eng.generate([Z.tokens(cfg, 3, 1), Z.tokens(cfg, 70, 2)], SamplingParams(temperature=1.0, max_new_tokens=300, seed=3))
    eng.sleep(False)
    for r in recs:
        z = Z.run_cut(eng, "x", r.prompt + r.out_tokens, [1000])[len(r.prompt) - 1 : -1]
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert (lp - torch.tensor(r.out_logprobs)).abs().median() < 0.1


# ------------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("shape", [dict(heads=4, kv_heads=2, dim=16, vdim=24), dict(heads=6, kv_heads=2, dim=128, vdim=128), dict(heads=3, kv_heads=3, dim=7, vdim=5)])
@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("size,keep", [(0, 0), (64, 0), (65, 1), (100, 64), (100, 65), (128, 130), (30, 7), (1, 20), (255, 3)])
@pytest.mark.parametrize("n", [1, 3, 40, 156, 256])
def test_one_key_far_away(shape, size, keep, n, dt):
    """The key stands just inside and just outside the window of the first and the last query, at the kept tokens' edge and at borders of pages."""
    for far in sorted({0, keep - 1, keep, 63, 64, 127, 128, 255 - size, 256 - size, 256 - n - size, 257 - n - size, 255} & set(range(256))):
        m = build(Z.attention(rot_dims=0, scale=2.0, size=size, keep=keep, source=0 if far % 3 == 1 and n < 256 else None, **shape), dt, DEV)
        p, b, kc, vc, want = Z.standout_case(m, 256, 64, far, n, DEV, dt, S.portion_tiles(m, dt))
        with torch.no_grad():
            got = S.attention(p, m, b, kc, vc, None, S.KeyValues(p, m))[:, : m.heads * m.vdim]
        assert (got.double().cpu() - want).abs().max() < (1e-4 if dt == F32 else 3e-2), far


@pytest.mark.parametrize("size,keep", [(0, 0), (1, 0), (33, 5), (64, 64), (100, 65), (128, 0), (300, 200)])
@pytest.mark.parametrize("shape", [(6, 2, 48, 40, 32, [1, 77, 5, 100, 17], [299, 0, 0, 29, 623]), (16, 4, 128, 128, 64, [1, 200, 128, 2, 1], [999, 0, 0, 127, 0]),
                                   (8, 1, 64, 96, 64, [300, 33], [0, 0]), (2, 2, 16, 256, 0, [300, 20, 1], [0, 480, 69]), (9, 3, 256, 8, 200, [70, 1], [3, 64]),
                                   (8, 1, 128, 128, 128, [1, 1, 1, 65], [127, 128, 1500, 300]), (4, 4, 64, 64, 30, [40, 200, 1], [300, 900, 9])])
@pytest.mark.parametrize("borrowed", [False, True])
def test_attention_kernels(shape, size, keep, borrowed):
    """Tensor-core kernels against the plain one; caches are equal, the prepared rows those of the module's statement."""
    H, G, dim, vdim, rd, lens, starts = shape
    torch.manual_seed(0)
    entry = Z.attention(heads=H, kv_heads=G, dim=dim, vdim=vdim, rot_dims=rd, scale=1.5 / math.sqrt(dim), size=size, keep=keep)
    m, source = build(entry, BF, DEV), None
    if borrowed:
        source, m = m, build({"mixer": dict(entry["mixer"], kv_from=0)}, BF, DEV)
    with torch.no_grad():
        m.offset.copy_(torch.randn(H, device=DEV) - 2)
    out = []
    order = sorted(range(len(lens)), key=lambda j: lens[j])
    for tiles in (False, True):
        torch.manual_seed(1)
        b, pages = batch(lens, starts, tiles=tiles)
        kc, vc = torch.randn(pages, G, 64, dim, device=DEV).to(BF), torch.randn(pages, G, 64, vdim, device=DEV).to(BF)
        p, kv = torch.randn(b.rows, m.in_width + 16, device=DEV).to(BF), None
        if borrowed:
            kv = S.KeyValues(torch.randn(b.rows, source.in_width, device=DEV).to(BF), source)
        if b.cu_q is not None and size:
            tiled = [j for j in order if lens[j] > X.PAGED_PORTION]
            cu = b.cu_ctx.tolist()
            Z.window_contexts(b, [lens[j] for j in tiled], [starts[j] for j in tiled], [b.ctx_slots[s:e] for s, e in zip(cu[:-1], cu[1:])], m)
        keep_fn = S.decode_tiles
        with torch.no_grad():
            if borrowed:
                S.attention(kv.p, source, b, kc, vc, None, kv)
                kv.gathered.clear()
            else:
                k, v = m.keys_values(p, b.positions)
            q = m.queries(p, b.positions)
            try:
                if not tiles:
                    S.decode_tiles = lambda *a: False
                y = S.attention(p, m, b, kc, vc, None, kv)[:, : H * vdim]
            finally:
                S.decode_tiles = keep_fn
        out.append((y, kc, vc))
        for t, off, n in ((q, m.q_off, H * dim),) + (() if borrowed else ((k, m.k_off, G * dim), (v, m.v_off, G * vdim))):
            assert rel(p[:, off : off + n], t.reshape(-1, n)) < 4e-3
    assert S.portion_tiles(m, BF) and rel(out[1][0], out[0][0]) < 8e-3
    assert torch.equal(out[0][1], out[1][1]) and torch.equal(out[0][2], out[1][2])


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("shape", [(3, 1, 15, 9, 6, 10, 4), (4, 2, 16, 8, 16, 5, 0), (2, 2, 128, 64, 64, 20, 30)])
def test_plain_attention_equals_the_statement(shape, dt):
    H, G, dim, vdim, rd, size, keep = shape
    m = build(Z.attention(heads=H, kv_heads=G, dim=dim, vdim=vdim, rot_dims=rd, size=size, keep=keep), dt, DEV)
    b, pages = batch([1, 4, 1], [70, 0, 3], tiles=False)
    kc, vc = torch.randn(pages, G, 64, dim, device=DEV).to(dt), torch.randn(pages, G, 64, vdim, device=DEV).to(dt)
    p = torch.randn(b.rows, m.in_width, device=DEV).to(dt)
    with torch.no_grad():
        cpu = X.TokenBatch(**{k: (v.cpu() if isinstance(v, torch.Tensor) else v) for k, v in b.__dict__.items()})
        want = S.attention(p.cpu().float(), build(Z.attention(heads=H, kv_heads=G, dim=dim, vdim=vdim, rot_dims=rd, size=size, keep=keep)), cpu, kc.cpu().float(), vc.cpu().float())
        keep_fn, S.decode_tiles = S.decode_tiles, lambda *a: False
        try:
            got = S.attention(p, m, b, kc, vc)
        finally:
            S.decode_tiles = keep_fn
    assert rel(got[:, : H * vdim], want[:, : H * vdim]) < (1e-5 if dt == F32 else 1e-2)


# ------------------------------------------------------------------------------------------------ feed-forwards, joins
@pytest.mark.parametrize("T", [1, 40, 300, 1500])
@pytest.mark.parametrize("spec,width", [(Z.moe(experts=14, identity=2, top=3, ff=40, shared=72), 264), (Z.moe(experts=64, identity=8, top=8, ff=64, shared=0), 256), (Z.moe(experts=5, identity=1, top=2, ff=7, shared=9), 61),
                                        (Z.moe(experts=8, identity=0, top=8, ff=24, shared=16), 64), (Z.moe(experts=2, identity=40, top=6, ff=56, shared=104), 320)])
def test_expert_kernels(spec, width, T):
    """Routing, identity outputs, placement, grouped products, gated shared unit and the join beside the module's statement."""
    class C2(Cfg):
        hidden_size = width
    torch.manual_seed(0)
    w = {k: v.to(F64) for k, v in O.below(Z.weights(Z.config([(Z.attention(), spec)], width=width), 5), "l0.mlp.").items()}
    h = torch.randn(T, width, dtype=F64).to(BF)
    ow, ls, nw = (torch.rand(width).to(BF).float() + 0.5 for _ in range(3))
    with torch.no_grad():
        want = O.rms(Z.module_weights(unit(spec, F32, "cpu", C2), w)(h.float()).double(), 1e-3) * ow.double() * ls.double()
    for dt, tol in ((F32, 1e-4), (BF, 0.02)):
        m = Z.module_weights(unit(spec, dt, DEV, C2), w)
        x = torch.ones(T, width, device=DEV)
        with torch.no_grad():
            x, g = Y.feed_forward(x, h.to(DEV, dt), m, ow.to(DEV, dt), 1.0, 1e-3, nw.to(DEV, dt), ls.to(DEV, dt))
        bad = ((x.double().cpu() - 1 - want).norm(dim=-1) / want.norm(dim=-1)) > tol      # (rows with a tie within rounding aside)
        assert bad.sum() <= (0 if dt == F32 else max(1, T // 100))
        assert rel(g, O.rms(x.double().cpu(), 1e-3) * nw.to(dt).double()) < (1e-5 if dt == F32 else 4e-3)
    assert all(int(c.abs().sum()) == 0 for c in Y._COUNTS.values())


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("rows", [1, 700])
@pytest.mark.parametrize("n", [1, 7, 40, 1000, 2048, 4096, 6144, 8192, 16384, 20000])
def test_poly_norm(n, rows, dt):
    torch.manual_seed(0)
    z, c = torch.randn(rows, n + 8, device=DEV).to(dt), torch.randn(4, device=DEV).to(dt)
    if n > 4096 and rows > 1:
        z = z[:40]
    want = O.poly_norm(z[:, :n].double(), c.double(), 1e-3)
    tail = z[:, n:].clone()
    Y.poly_norm_(z, c, n, 1e-3)
    assert rel(z[:, :n], want) < (1e-5 if dt == F32 else 4e-3) and torch.equal(z[:, n:], tail)


@pytest.mark.parametrize("dt,tol", [(F32, 1e-5), (BF, 1e-2)])
@pytest.mark.parametrize("bigram", [(13, 5, 3), None])
@pytest.mark.parametrize("d", [8, 7, 1024, 1500, 2048, 4096, 8192, 9001])
def test_start_and_shift_kernels_over_steps(bigram, d, dt, tol):
    start_and_shift(bigram, d, DEV, dt, tol)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("d", [37, 264, 2048, 4096])
@pytest.mark.parametrize("lens", [[1, 1, 700], [5, 900, 2000], [1] * 650, [3000, 3000]])
def test_shift_of_many_rows(lens, d, dt):
    """Runs of rows per CTA: with expert rows and factors, beside the plain statement of the same operator."""
    torch.manual_seed(0)
    T, k = sum(lens), 3
    b = pieces(lens, [7 * (j % 2) for j in range(len(lens))], list(range(1, len(lens) + 1)), [0] * T, DEV, torch.int32)
    carry = Y.Carry(len(lens) + 1, 2, d, False, DEV)
    carry.state.normal_()
    x, y, h, also = (torch.randn(T, d, device=DEV).to(t) for t in (F32, dt, dt, dt))
    w, ls, nw, s = (torch.rand(d, device=DEV).to(dt) for _ in range(4))
    rows, wt, f1, f2 = torch.randint(-1, T, (T, k), device=DEV, dtype=torch.int32), torch.rand(T, k, device=DEV), torch.rand(T, device=DEV), torch.rand(T, device=DEV)
    counts = torch.ones(6, dtype=torch.int32, device=DEV)
    carry.next.copy_(carry.state)      # (a step fills all places)
    before = carry.state.clone()
    gx, gh = Y.join(x.clone(), y, w, 1.0, 1e-3, nw, (rows, wt, counts), also, f1, h, f2, ls, Y.Shift(s, 1, carry, b))
    carry.commit(b)
    v = (torch.where(rows[..., None] >= 0, y[rows.clamp(min=0).long()].double(), 0.0) * wt[..., None].double()).sum(1) + also.double() * f1[:, None] + h.double() * f2[:, None]
    want = x.double() + O.rms(v, 1e-3) * w.double() * ls.double()
    n = O.rms(want, 1e-3) * nw.double()
    prev, at = torch.cat([n[:1], n[:-1]]), 0
    for j, L_ in enumerate(lens):
        prev[at] = before[j + 1, 1].double() if j % 2 else 0.0
        at += L_
        assert rel(carry.state[j + 1, 1], n[at - 1]) < 1e-5
    assert torch.equal(carry.state[:, 0], before[:, 0]) and int(counts.sum()) == 0
    assert rel(gx, want) < 1e-5 and rel(gh, n + (prev - n) * s.double()) < (1e-5 if dt == F32 else 4e-3)


def test_presets_generate_with_captured_steps():
    m = build_model(preset("tiny-zonidra"), device=DEV, dtype=BF, seed=1)
    prompts = [Z.tokens({"vocab": 264}, n, n) for n in (5, 70, 129, 1)]
    outs = []
    for graphs in (True, False):
        eng = Z.engine(m, pages=40, block_size=64, use_cuda_graphs=graphs)
        outs.append([r.out_tokens for r in eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))])
        assert bool(eng._graphs) == graphs
    assert outs[0] == outs[1]
