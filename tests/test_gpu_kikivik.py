"""Kikivik (pre-norm layer-list models) on the GPU: the native kernels of both precisions against the float64 oracle, the tensor-core forms
against the plain kernels at many shapes, and generation through captured decode steps."""

import math

import kikivik_cases as K
import kikivik_oracle as O
import pytest
import torch
from test_gpu_redarax import batch
from test_kikivik import Cfg, build, unit

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import preset
from rl_b200.models.transformer import build_model
from rl_b200.ops import engine_ops as E
from rl_b200.ops import layer_ops as Y
from rl_b200.ops import lib as L
from rl_b200.ops import mixer_ops as X
from rl_b200.ops import sequence_ops as S

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32, F64 = torch.bfloat16, torch.float32, torch.float64
# sizes that every tensor-core kernel takes, wide enough for the weight-streaming product; chunks across and inside tiles of 64 and 128 keys
TILED = K.config([(K.attention(heads=6, kv_heads=2, dim=48, vdim=128, rot_dims=32, scale=0.2, size=100), K.moe(experts=16, top=3, ff=40, shared=72)),
                  (K.latent(heads=6, dim=48, rot_dim=32, vdim=40, kv_rank=72, q_rank=136), K.dense(ff=136)),
                  (K.attention(heads=4, kv_heads=2, dim=128, vdim=128, rot_dims=128, scale=0.1, size=70), None),
                  (K.latent(heads=20, dim=16, rot_dim=8, vdim=24, kv_rank=24, q_rank=40), K.moe(experts=8, top=1, ff=64, shared=0)),
                  (K.attention(heads=8, kv_heads=2, dim=64, vdim=128, rot_dims=20, factor=0, scale=0.2, size=0), K.dense(ff=72))], width=264, vocab=200)
CASES = dict(K.CASES, tiled=TILED)


@pytest.fixture(autouse=True)
def _clean(native_lib):
    yield
    assert L.check_status() == 0


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request, tmp_path_factory):
    cfg = CASES[request.param]
    w = K.weights(cfg, seed=7)
    path = tmp_path_factory.mktemp(request.param)
    return cfg, w, {dt: K.load(cfg, w, path, DEV, dt) for dt in (F32, BF)}


def rel(a, b):
    return ((a.double().cpu() - b.double().cpu()).norm() / b.double().cpu().norm()).item()


def gaps(got, want):
    d = got.double().cpu() - want
    d = d - d.mean(-1, keepdim=True)
    s = want - want.mean(-1, keepdim=True)
    return d.pow(2).mean(-1).sqrt() / s.pow(2).mean().sqrt()


def close(cfg, w, toks, got, dt):
    """fp32: every position. bf16: the median, and every position up to the first one where a router's choice is within a rounding."""
    g = gaps(got, K.oracle(cfg, w, toks))
    if dt == F32:
        return g.max() < 5e-4
    flip = K.close_routes(cfg, w, toks, 0.05).nonzero()
    n = int(flip[0]) if len(flip) else len(toks)
    return g.median() < 0.08 and (n == 0 or g[:n].max() < 0.3)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [17, 2, 33, 1], [130, 1], [100, 70, 1]])
def test_portions_equal_the_oracle(case, dt, cuts):
    cfg, w, models = case
    toks = K.tokens(cfg, 90 if cuts == [1] else 220)
    eng = K.engine(models[dt], block_size=64, pages=6)
    assert close(cfg, w, toks, K.run_cut(eng, "a", toks, cuts), dt)


@pytest.mark.parametrize("dt", [F32, BF])
def test_mixed_batches_and_reused_pages(case, dt):
    cfg, w, models = case
    seqs = {f"r{i}": K.tokens(cfg, n, seed=i) for i, n in enumerate([150, 1, 33, 17, 90, 2, 160, 16])}
    steps = K.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = K.engine(models[dt], pages=K.live_pages(steps, 32), block_size=32)
    got = K.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert close(cfg, w, t, got[r], dt), r
    assert eng.sched.num_free_blocks == eng.num_blocks


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation(case, graphs):
    """fp32: the tokens the oracle picks, through the scheduler, portions, shared pages and (captured) multi-step decode windows."""
    cfg, w, models = case
    prompts = [K.tokens(cfg, n, seed=n) for n in (1, 5, 64, 65, 140, 5)]
    prompts[5] = list(prompts[1])
    prompts.append(prompts[4][:129])
    eng = K.engine(models[F32], pages=20, block_size=64, requests=3, max_prefill_tokens=48, use_cuda_graphs=graphs)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=20))
    for p, r in zip(prompts, recs):
        z = K.oracle(cfg, w, p + r.out_tokens)[len(p) - 1 : -1]
        top = z.topk(2, -1)
        clear = top[0][:, 0] - top[0][:, 1] > 1e-2
        assert (top[1][:, 0] == torch.tensor(r.out_tokens))[clear].all()
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert torch.allclose(lp, torch.tensor(r.out_logprobs, dtype=F64), atol=5e-3)
    assert bool(eng._graphs) == graphs


def test_long_decoding_keeps_to_the_prefill(case):
    """300 decoded tokens (captured steps, windows, page and chunk borders): the log-probabilities are those of one prefill of the same tokens."""
    cfg, w, models = case
    eng = K.engine(models[BF], pages=14, block_size=64, requests=2, use_cuda_graphs=True)
    recs = eng.generate([K.tokens(cfg, 3, 1), K.tokens(cfg, 70, 2)], SamplingParams(temperature=1.0, max_new_tokens=300, seed=3))
    eng.sleep(False)
    for r in recs:
        z = K.run_cut(eng, "x", r.prompt + r.out_tokens, [1000])[len(r.prompt) - 1 : -1]
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert (lp - torch.tensor(r.out_logprobs)).abs().median() < 0.1


# ------------------------------------------------------------------------------------------------ attention
@pytest.mark.parametrize("shape", [dict(heads=4, kv_heads=2, dim=16, vdim=24), dict(heads=6, kv_heads=2, dim=128, vdim=128), dict(heads=3, kv_heads=3, dim=7, vdim=5)])
@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("size,far", [(0, 0), (0, 127), (64, 63), (64, 64), (64, 191), (100, 99), (100, 100), (100, 199), (100, 200), (128, 0), (128, 127), (128, 128), (255, 254), (255, 255),
                                      (256, 0), (256, 255), (7, 250)])
@pytest.mark.parametrize("n", [1, 3, 40, 56, 156, 256])
def test_one_key_far_away(shape, size, far, n, dt):
    m = build(K.attention(rot_dims=0, factor=0, scale=2.0, size=size, v_mix=False, **shape), dt, DEV)
    p, b, kc, vc, want = K.standout_case(m, 256, 64, far, n, DEV, dt, S.portion_tiles(m, dt))
    with torch.no_grad():
        got = S.attention(p, m, b, kc, vc)[:, : m.heads * m.vdim]
    d = (got.double().cpu() - want).abs().max()
    assert d < (1e-4 if dt == F32 else 3e-2)


def chunked(b, lens, starts, m):
    """Adds to ``b`` (see ``batch``) the contexts from the border of a chunk on, as the engine builds them."""
    if b.cu_q is None or not m.chunk:
        return b
    order = [j for j in sorted(range(len(lens)), key=lambda j: lens[j]) if lens[j] > X.PAGED_PORTION]
    lo = [starts[j] // m.chunk * m.chunk for j in order]
    at, cut, cu = b.cu_ctx.tolist(), [], [0]
    for k, j in enumerate(order):
        cut.append(b.ctx_slots[at[k] + lo[k] : at[k + 1]])
        cu.append(cu[-1] + cut[-1].numel())
    b.chunk_ctx[m.chunk] = (torch.tensor(cu, dtype=torch.int32, device=DEV), torch.cat(cut), all(starts[j] == s for j, s in zip(order, lo)))
    return b


@pytest.mark.parametrize("size", [0, 1, 33, 64, 100, 128, 300])
@pytest.mark.parametrize("shape", [(6, 2, 48, 40, 32, [1, 77, 5, 100, 17], [299, 0, 0, 29, 623]), (16, 4, 128, 128, 64, [1, 200, 128, 2, 1], [999, 0, 0, 127, 0]),
                                   (8, 1, 64, 96, 64, [300, 33], [0, 0]), (2, 2, 16, 256, 0, [300, 20, 1], [0, 480, 69]), (9, 3, 256, 8, 200, [70, 1], [3, 64]),
                                   (8, 1, 128, 128, 128, [1, 1, 1, 65], [127, 128, 1500, 300]), (4, 4, 64, 64, 30, [40, 200, 1], [300, 100, 9])])
def test_attention_kernels(shape, size):
    """Tensor-core kernels against the plain one, with mixed values; caches are equal, the prepared rows those of the module's statement."""
    H, G, dim, vdim, rd, lens, starts = shape
    torch.manual_seed(0)
    m = build(K.attention(heads=H, kv_heads=G, dim=dim, vdim=vdim, rot_dims=rd, scale=1.5 / math.sqrt(dim), size=size), BF, DEV)
    with torch.no_grad():
        m.q_norm.uniform_(0.5, 1.5), m.k_norm.uniform_(0.5, 1.5), m.v_share.fill_(0.3)
    out = []
    for tiles in (False, True):
        torch.manual_seed(1)
        b, pages = batch(lens, starts, tiles=tiles)
        chunked(b, lens, starts, m)
        kc, vc = torch.randn(pages, G, 64, dim, device=DEV).to(BF), torch.randn(pages, G, 64, vdim, device=DEV).to(BF)
        p, first = torch.randn(b.rows, m.in_width + 16, device=DEV).to(BF), torch.randn(b.rows, G * vdim + 6, device=DEV).to(BF)[:, 2 : 2 + G * vdim]
        keep = S.decode_tiles
        with torch.no_grad():
            q, k, v = m.qkv(p, b.positions, first)
            try:
                if not tiles:
                    S.decode_tiles = lambda *a: False
                y = S.attention(p, m, b, kc, vc, first)[:, : H * vdim]
            finally:
                S.decode_tiles = keep
        out.append((y, kc, vc))
        for t, off, n in ((q, m.q_off, H * dim), (k, m.k_off, G * dim), (v, m.v_off, G * vdim)):
            assert rel(p[:, off : off + n], t.reshape(-1, n)) < 4e-3
    assert S.portion_tiles(m, BF) and rel(out[1][0], out[0][0]) < 6e-3
    assert torch.equal(out[0][1], out[1][1]) and torch.equal(out[0][2], out[1][2])


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("rd", [0, 2, 6, 12, 14])
def test_preparation_of_odd_sizes(rd, dt):
    m = build(K.attention(heads=3, kv_heads=1, dim=15, vdim=9, rot_dims=rd), dt, DEV)
    b, pages = batch([1, 4], [70, 0], tiles=False)
    kc, vc = torch.zeros(pages, 1, 64, 15, device=DEV, dtype=dt), torch.zeros(pages, 1, 64, 9, device=DEV, dtype=dt)
    p, first = torch.randn(b.rows, m.in_width, device=DEV).to(dt), torch.randn(b.rows, 9, device=DEV).to(dt)
    q, k, v = m.qkv(p, b.positions, first)
    S.attention(p, m, b, kc, vc, first)
    for t, off, n in ((q, m.q_off, 45), (k, m.k_off, 15), (v, m.v_off, 9)):
        assert rel(p[:, off : off + n], t.reshape(-1, n)) < (1e-5 if dt == F32 else 4e-3)
    assert torch.equal(kc.view(-1, 15)[b.slots], p[:, m.k_off : m.k_off + 15]) and torch.equal(vc.view(-1, 9)[b.slots], p[:, m.v_off : m.v_off + 9])


@pytest.mark.parametrize("shape", [(6, 48, 32, 40, 72, 136, [1, 77, 5, 100, 17], [299, 0, 0, 29, 623]), (20, 16, 8, 24, 24, 40, [1, 200, 2, 1], [999, 0, 127, 0]),
                                   (16, 128, 64, 128, 512, 768, [1, 1, 130, 1], [640, 63, 200, 64])])
def test_latent_kernels(shape):
    """Tensor-core kernels against the plain one, and the fp32 plain one against the module's statement."""
    H, dim, rd, vdim, R, Q, lens, starts = shape

    class C2(Cfg):
        hidden_size = 64
    outs = {}
    for dt, tiles in ((F32, False), (BF, False), (BF, True)):
        m = build(K.latent(heads=H, dim=dim, rot_dim=rd, vdim=vdim, kv_rank=R, q_rank=Q, scale=1.5 / math.sqrt(dim + rd)), dt, DEV, C2)
        torch.manual_seed(1)
        with torch.no_grad():
            for prm in (m.q_up, m.kv_up):
                prm.copy_(torch.randn(prm.shape, device=DEV).to(BF) / math.sqrt(prm.shape[1]))
            m.q_norm.copy_((torch.rand(Q, device=DEV) + 0.5).to(BF)), m.kv_norm.copy_((torch.rand(R, device=DEV) + 0.5).to(BF))
            b, pages = batch(lens, starts, tiles=tiles)
            cache = torch.randn(pages, 64, m.latent_width, device=DEV).to(BF).to(dt)
            p = torch.randn(b.rows, m.in_width, device=DEV).to(BF).to(dt)
            p[:, Q : m.lat_off] = 0
            keep = X.decode_tiles
            try:
                if not tiles:
                    X.decode_tiles = lambda *a: False
                y = X.latent_attention(p.clone(), m, b, cache)[:, : H * vdim]
                if dt == F32:
                    cpu = {k: (v.cpu() if isinstance(v, torch.Tensor) else v) for k, v in b.__dict__.items()}
                    want = X.latent_attention(p.cpu(), m.to("cpu"), X.TokenBatch(**cpu), cache.cpu())[:, : H * vdim]
                    assert rel(y, want) < 1e-5
            finally:
                X.decode_tiles = keep
        outs[dt, tiles] = y
    assert X.portion_tiles(m, BF) and rel(outs[BF, True], outs[BF, False]) < 1e-2 and rel(outs[BF, False], outs[F32, False]) < 2e-2


@pytest.mark.parametrize("chunk", [0, 1, 64, 100, 128, 1000])
@pytest.mark.parametrize("bs", [16, 64, 128])
@pytest.mark.parametrize("splits", [1, 5])
def test_paged_decode_sees_its_chunk(chunk, bs, splits):
    G, H, D = 2, 8, 128
    lens = torch.tensor([1, 64, 65, 100, 101, 128, 129, 700, 1000, 0], dtype=torch.int32, device=DEV)
    n = -(-1000 // bs)
    kc, vc = (torch.randn(n * 10, G, bs, D, device=DEV).to(BF) for _ in range(2))
    q = torch.randn(10, H * D, device=DEV).to(BF)
    bt = torch.randperm(n * 10, device=DEV).view(10, n).int()
    got = E.paged_decode(q, kc, vc, bt, lens, H, G, D, scale=0.2, num_splits=splits, chunk=chunk)
    want = E._paged_decode_gather(q, kc, vc, bt, lens, H, G, D, 0.2, torch.empty_like(got), chunk=chunk)
    assert rel(got, want) < 1e-2


# ------------------------------------------------------------------------------------------------ feed-forwards, products, joins
@pytest.mark.parametrize("T", [1, 40, 300, 1500])
@pytest.mark.parametrize("spec,width", [(K.moe(experts=16, top=3, ff=40, shared=72), 264), (K.moe(experts=64, top=8, ff=64, shared=0), 256), (K.moe(experts=5, top=2, ff=7, shared=9), 61),
                                        (K.moe(experts=8, top=8, ff=24, shared=16), 64), (K.moe(experts=10, top=1, ff=56, shared=104), 320)])
def test_expert_kernels(spec, width, T):
    """Routing, placement, weighted grouped products, shared unit and the join beside the module's statement; fp32 beside float64."""
    class C2(Cfg):
        hidden_size = width
    torch.manual_seed(0)
    w = {k: v.to(F64) for k, v in O.below(K.weights(K.config([(K.latent(), spec)], width=width), 5), "l0.mlp.").items()}
    h = torch.randn(T, width, dtype=F64).to(BF)
    nw = torch.rand(width) + 0.5
    with torch.no_grad():
        want = K.module_weights(unit(spec, F32, "cpu", C2), w)(h.float()).double()
    for dt, tol in ((F32, 1e-4), (BF, 0.02)):
        m = K.module_weights(unit(spec, dt, DEV, C2), w)
        x = torch.ones(T, width, device=DEV)
        with torch.no_grad():
            g = Y.feed_forward_(x, h.to(DEV, dt), m, None, 1.0, 1e-3, nw.to(DEV, dt))
        bad = ((x.double().cpu() - 1 - want).norm(dim=-1) / want.norm(dim=-1)) > tol      # (rows with a tie within rounding aside)
        assert bad.sum() <= (0 if dt == F32 else max(1, T // 100))
        assert rel(g, O.rms(x.double().cpu(), 1e-3) * nw.to(dt).double()) < (1e-5 if dt == F32 else 4e-3)
    assert all(int(c.abs().sum()) == 0 for c in Y._COUNTS.values())


@pytest.mark.parametrize("M,N,K_", [(1, 64, 64), (5, 400, 328), (64, 2048, 4096), (300, 1104, 320), (257, 96, 72), (130, 38, 61), (3, 200, 520)])
@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("limit", [None, 1.3])
def test_gated_products(M, N, K_, dt, limit):
    torch.manual_seed(0)
    a, w = torch.randn(M, K_, device=DEV).to(dt), (torch.randn(N, K_, device=DEV) * 1.5 / math.sqrt(K_)).to(dt)
    ref = (a.double() @ w.double().T).float().cpu()
    assert rel(Y.gated_linear(a, w, limit), Y.gated_ref(ref, limit)) < (1e-5 if dt == F32 else 5e-3)


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("d", [37, 264, 2048, 4096, 9000])
def test_start_and_joins(d, dt):
    torch.manual_seed(0)
    nw, table = torch.randn(d, device=DEV).to(dt), torch.randn(50, d, device=DEV).to(dt)
    for rows in (3, 700):
        x, y, z = torch.randn(rows, d, device=DEV), torch.randn(rows, d, device=DEV).to(dt), torch.randn(rows, d, device=DEV).to(dt)
        for also in (None, z):
            want = x.double() + y.double() + (0 if also is None else z.double())
            x1 = x.clone()
            h = Y.add_normed_(x1, y, None, 1.0, 1e-3, nw, also=also)
            assert rel(x1, want) < 1e-6 and rel(h, O.rms(want, 1e-3) * nw.double()) < (1e-6 if dt == F32 else 4e-3)
        ids = torch.randint(0, 50, (rows,), device=DEV, dtype=torch.int32)
        want = table[ids.long()].double() * 1.7
        for norm in (nw, None):
            x1, h = Y.embed(ids, table, 1.7, norm, 1e-3)
            assert rel(x1, want) < 1e-6 and rel(h, want if norm is None else O.rms(want, 1e-3) * nw.double()) < (1e-6 if dt == F32 else 4e-3)
        z1 = z.clone()
        Y.group_norm_(z1, nw, 1, 1e-3)
        assert rel(z1, O.rms(z.double(), 1e-3) * nw.double()) < (1e-6 if dt == F32 else 4e-3)


def test_presets_generate_with_captured_steps():
    m = build_model(preset("tiny-kikivik"), device=DEV, dtype=BF, seed=1)
    prompts = [K.tokens({"vocab": 264}, n, n) for n in (5, 70, 129, 1)]
    outs = []
    for graphs in (True, False):
        eng = K.engine(m, pages=40, block_size=64, use_cuda_graphs=graphs)
        outs.append([r.out_tokens for r in eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))])
        assert bool(eng._graphs) == graphs
    assert outs[0] == outs[1]
