"""Gadarax (layer-list models) on the GPU: the native kernels of both precisions against the float64 oracle, the tensor-core forms
against the plain kernels at many shapes, and generation through captured decode steps."""

import math

import gadarax_cases as G
import pytest
import torch
from test_gadarax import Cfg, standout_case

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import preset
from rl_b200.models.mixers import LatentAttentionMixer, RetentionMixer
from rl_b200.models.transformer import build_model
from rl_b200.ops import lib as L
from rl_b200.ops import mixer_ops as X

pytestmark = pytest.mark.gpu
DEV = "cuda"
BF, F32 = torch.bfloat16, torch.float32
# a case whose sizes every tensor-core kernel takes, and wide enough for the weight-streaming GEMM
TILED = G.config([G.latent(heads=4, dim=32, rot_dim=16, vdim=40, kv_rank=72, scaling=G.YARN), G.retention(heads=3, dim=40, vdim=32, rot_dims=24),
                  G.latent(heads=18, dim=16, rot_dim=8, vdim=16, kv_rank=136)], width=264, vocab=200, ff=[136, 320, None], loop={"start": 1, "stop": 3, "times": 2})
CASES = dict(G.CASES, tiled=TILED)


@pytest.fixture(autouse=True)
def _clean(native_lib):
    yield
    assert L.check_status() == 0


@pytest.fixture(scope="module", params=sorted(CASES))
def case(request, tmp_path_factory):
    cfg = CASES[request.param]
    w = G.weights(cfg, seed=7, sharp=1.5)
    path = tmp_path_factory.mktemp(request.param)
    return cfg, w, {dt: G.load(cfg, w, path, DEV, dt) for dt in (F32, BF)}


def rel(a, b):
    return ((a.float() - b.float()).norm() / b.float().norm()).item()


TOLS = {F32: 2e-5, BF: 0.06}


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [17, 2, 33, 1], [130, 1]])
def test_portions_equal_the_oracle(case, dt, cuts):
    cfg, w, models = case
    toks = G.tokens(cfg, 90 if cuts == [1] else 200)
    eng = G.engine(models[dt], block_size=64, pages=6)
    assert G.gap(G.run_cut(eng, "a", toks, cuts), G.oracle(cfg, w, toks)) < TOLS[dt]


@pytest.mark.parametrize("dt", [F32, BF])
def test_mixed_batches_and_reused_pages(case, dt):
    cfg, w, models = case
    seqs = {f"r{i}": G.tokens(cfg, n, seed=i) for i, n in enumerate([150, 1, 33, 17, 90, 2, 160, 16])}
    steps = G.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = G.engine(models[dt], pages=G.live_pages(steps, 32), block_size=32)
    got = G.run_schedule(eng, steps, seqs)
    alone = G.engine(models[dt], pages=8, block_size=64)
    for r, t in seqs.items():
        assert G.gap(got[r], G.oracle(cfg, w, t)) < TOLS[dt], r
        assert G.gap(got[r], G.run_cut(alone, r, t, [1000]).double()) < TOLS[dt], r
    assert eng.sched.num_free_blocks == eng.num_blocks


@pytest.mark.parametrize("graphs", [True, False])
def test_greedy_generation(case, graphs):
    """fp32: the tokens the oracle picks, through the scheduler, chunked prefill and (captured) multi-step decode windows."""
    cfg, w, models = case
    prompts = [G.tokens(cfg, n, seed=n) for n in (1, 5, 64, 65, 40, 5)]
    prompts[5] = list(prompts[1])
    eng = G.engine(models[F32], pages=20, block_size=64, requests=3, max_prefill_tokens=48, use_cuda_graphs=graphs)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=20))
    for p, r in zip(prompts, recs):
        z = G.oracle(cfg, w, p + r.out_tokens)[len(p) - 1 : -1]
        assert z.argmax(-1).tolist() == r.out_tokens
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert torch.allclose(lp, torch.tensor(r.out_logprobs, dtype=torch.float64), atol=1e-3)
    assert bool(eng._graphs) == graphs


def test_long_decoding_keeps_to_the_prefill(case):
    """300 decoded tokens (captured steps, windows, page borders): the log-probabilities are those of one prefill of the same tokens."""
    cfg, w, models = case
    eng = G.engine(models[BF], pages=14, block_size=64, requests=2, use_cuda_graphs=True)
    recs = eng.generate([G.tokens(cfg, 3, 1), G.tokens(cfg, 70, 2)], SamplingParams(temperature=1.0, max_new_tokens=300, seed=3))
    eng.sleep(False)
    for r in recs:
        z = G.run_cut(eng, "x", r.prompt + r.out_tokens, [1000])[len(r.prompt) - 1 : -1]
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert (lp - torch.tensor(r.out_logprobs)).abs().mean() < 0.05


@pytest.mark.parametrize("dt", [F32, BF])
@pytest.mark.parametrize("far", [0, 1, 63, 64, 65, 127, 128, 191, 255])
@pytest.mark.parametrize("n", [1, 3, 40, 256])
def test_one_key_far_away(far, n, dt):
    T, bs = 256, 64
    m, p, b, cache, want = standout_case(T, bs, far, n, DEV, dt, heads=3, dim=16, rot_dim=8, vdim=24, rank=72)
    X.latent_attention_(p, m, b, cache)
    got = p[:, m.mix_off : m.mix_off + m.heads * m.vdim].float().cpu()
    rows = [i for i in range(n) if T - n + i >= far]
    assert rel(got[rows], want[rows]) < (1e-5 if dt == F32 else 8e-3)
    hidden = [i for i in range(n) if T - n + i < far]
    assert not hidden or rel(got[hidden], want[hidden]) > 0.3


# ------------------------------------------------------------------------------------------------ tensor-core forms against the plain kernels
def latent_outputs(H, dim, rot, vdim, R, lens, news, bs):
    torch.manual_seed(0)
    spec = G.latent(heads=H, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=R, scaling=dict(factor=4.0, fast=32.0, slow=1.0, original=1024))["mixer"]
    m = LatentAttentionMixer(spec, Cfg, BF, DEV)
    with torch.no_grad():
        m.kv_up.normal_(std=1 / math.sqrt(R)), m.kv_norm.uniform_(0.5, 1.5)
    pages = [-(-n // bs) for n in lens]
    free = torch.randperm(sum(pages) + 3).tolist()
    own = [[free.pop() for _ in range(n)] for n in pages]
    cache = torch.zeros(sum(pages) + 3, bs, m.latent_width, dtype=BF, device=DEV)
    cache[..., : R + rot] = torch.randn(cache.shape[0], bs, R + rot, device=DEV).to(BF)
    order = sorted(range(len(lens)), key=lambda j: news[j])
    new = [news[j] for j in order]
    pos = torch.cat([torch.arange(lens[j] - news[j], lens[j]) for j in order]).int()
    slot = lambda j, lo: torch.tensor([own[j][t // bs] * bs + t % bs for t in range(lo, lens[j])])  # noqa: E731
    slots = torch.cat([slot(j, lens[j] - news[j]) for j in order]).to(DEV)
    bt = torch.zeros(len(lens), max(pages) + 1, dtype=torch.int32)
    for k, j in enumerate(order):
        bt[k, : pages[j]] = torch.tensor(own[j])
    bt = bt[torch.repeat_interleave(torch.arange(len(lens)), torch.tensor(new))].to(DEV)
    p = torch.randn(len(pos), m.in_width + 24, device=DEV).to(BF)

    def run(tiles, plain):
        tl = [k for k, n in enumerate(new) if n > X.PAGED_PORTION] if tiles else []
        n = sum(new[: tl[0]]) if tl else len(pos)
        b = X.TokenBatch(ids=None, positions=pos.to(DEV), slots=slots, n_single=sum(x == 1 for x in new), n_paged=n, block_table=bt[:n],
                         seq_lens=(pos[:n] + 1).to(DEV), max_ctx=max(lens))
        if tl:
            cu = torch.zeros(2, len(tl) + 1, dtype=torch.int32)
            cu[0, 1:] = torch.tensor([new[k] for k in tl]).cumsum(0)
            cu[1, 1:] = torch.tensor([lens[order[k]] for k in tl]).cumsum(0)
            b.cu_q, b.cu_ctx = cu.to(DEV)
            b.q_tiles, b.ctx_slots = sum(-(-new[k] // 128) for k in tl), torch.cat([slot(order[k], 0) for k in tl]).to(DEV)
        q, c = p.clone(), cache.clone()
        keep = X.decode_tiles
        try:
            if plain:
                X.decode_tiles = lambda *a: False
            X.latent_attention_(q, m, b, c)
        finally:
            X.decode_tiles = keep
        return q[:, m.mix_off : m.mix_off + H * vdim], c

    assert X.decode_tiles(p, m, bs) and X.portion_tiles(m, BF)
    return run(False, True), run(False, False), run(True, False)


@pytest.mark.parametrize("shape", [(9, 32, 24, 40, 136, [300, 77, 5, 129, 640], [1, 77, 5, 100, 17], 64),
                                   (16, 128, 64, 128, 512, [1000, 200, 130, 129, 1], [1, 200, 128, 2, 1], 64),
                                   (4, 48, 8, 40, 72, [300, 77, 70], [1, 77, 33], 64),
                                   (40, 64, 32, 96, 256, [300, 1000, 70], [300, 1, 33], 32),
                                   (3, 16, 24, 24, 200, [300, 500, 70], [300, 20, 1], 128),
                                   (20, 96, 64, 192, 384, [300, 500, 70], [300, 20, 1], 16),
                                   (2, 128, 64, 256, 512, [300, 500, 70], [300, 20, 1], 16),
                                   (1, 16, 8, 8, 8, [64, 65, 2], [64, 1, 2], 64)])
def test_latent_kernels(shape):
    (plain, cache), (dec, c1), (tiles, c2) = latent_outputs(*shape)
    assert rel(dec, plain) < 6e-3 and rel(tiles, plain) < 6e-3
    assert torch.equal(cache, c1) and torch.equal(cache, c2)


@pytest.mark.parametrize("H,dim,vdim,rd,lens,starts,decay", [
    (5, 64, 48, 64, [1, 2, 100, 300, 128, 1], [5, 0, 77, 0, 128, 0], None), (4, 128, 128, 128, [1, 129, 1000], [0, 0, 300], None),
    (2, 256, 256, 256, [1, 129, 400], [9, 0, 300], None), (3, 40, 24, 12, [1, 17, 140, 3], [9, 0, 300, 4], None),
    (5, 72, 136, 72, [260, 64], [0, 64], [1.0, 0.5, 0.25, 0.999, 0.9]), (2, 8, 8, 0, [5, 1], [3, 0], [0.75, 0.5])])
def test_retention_kernels(H, dim, vdim, rd, lens, starts, decay):
    """Chunked and single-step kernels against the token-by-token kernel: the states agree to fp32 rounding."""
    torch.manual_seed(1)
    m = RetentionMixer(G.retention(heads=H, dim=dim, vdim=vdim, rot_dims=rd, decay=decay or [1 - 2.0 ** -(2 + i % 9) for i in range(H)])["mixer"], Cfg, BF, DEV)
    order = sorted(range(len(lens)), key=lambda j: lens[j])
    new = [lens[j] for j in order]
    pos = torch.cat([torch.arange(starts[j], starts[j] + lens[j]) for j in order]).int().to(DEV)
    ns = sum(n == 1 for n in new)
    b = X.TokenBatch(ids=None, positions=pos, slots=None, n_single=ns, n_paged=0, block_table=None, seq_lens=None,
                     state_rows=torch.randperm(len(new) + 3)[: len(new)].to(DEV))
    if ns < len(new):
        b.cu = torch.tensor([0] + torch.tensor(new[ns:]).cumsum(0).tolist(), dtype=torch.int32, device=DEV)
        b.piece_chunk, b.chunk_row, b.chunk_rows = (t.to(DEV) for t in X.chunk_lists(new[ns:]))
    p = torch.randn(len(pos), m.in_width + 40, device=DEV).to(BF)
    S = torch.randn(len(new) + 3, H, dim, vdim, device=DEV)
    out = []
    for plain in (True, False):
        q, s = p.clone(), S.clone()
        X.retention_(q, m, b, s, plain=plain)
        out.append((q[:, m.mix_off : m.mix_off + H * vdim], s))
    (want, Sw), (got, Sg) = out
    assert rel(got, want) < 1e-3 and (Sg - Sw).abs().max() < 1e-4 * Sw.abs().max()
    untouched = [r for r in range(len(new) + 3) if r not in b.state_rows.tolist()]
    assert torch.equal(Sg[untouched], S[untouched])


@pytest.mark.parametrize("M,N,K,act", [(1, 64, 64, 32), (5, 400, 328, 200), (64, 2048, 4096, 512), (300, 1104, 320, 800), (257, 96, 72, 96), (130, 37, 61, 8), (3, 200, 520, 0)])
@pytest.mark.parametrize("dt", [F32, BF])
def test_products(M, N, K, act, dt):
    """All three product kernels (plain, weight-streaming, tiled) with both epilogues, beside an fp32 statement."""
    torch.manual_seed(0)
    a, w = torch.randn(M, K, device=DEV).to(dt), (torch.randn(N, K, device=DEV) / math.sqrt(K)).to(dt)
    tol = 1e-5 if dt == F32 else 4e-3
    ref = (a.double() @ w.double().T).float()
    sq = ref.clone()
    sq[:, act:] = torch.relu(sq[:, act:]) ** 2
    assert rel(X.in_proj(a, w, act), sq) < tol
    from rl_b200.models.mixers import DynamicTanh

    n = DynamicTanh(N, dt, DEV)
    with torch.no_grad():
        n.weight.normal_(), n.bias.normal_(), n.alpha.fill_(0.7)
        for e, step in ((torch.randn(M, N, device=DEV), torch.randn(3, N, device=DEV).to(dt)[1]), (None, None)):
            x = torch.randn(M, N, device=DEV) * torch.logspace(-4, 1, N, device=DEV)     # tanh near zero and saturated
            want = x + ref + (e if e is not None else 0) + (step.float() if step is not None else 0)
            h = X.out_proj_(x, a, w, e, step, n)
            assert rel(x, want) < 1e-5
            assert rel(h, torch.tanh(n.alpha.float() * want) * n.weight.float() + n.bias.float()) < tol


def test_presets_generate_with_captured_steps():
    m = build_model(preset("tiny-gadarax"), device=DEV, dtype=BF, seed=1)
    prompts = [G.tokens({"vocab": 264}, n, n) for n in (5, 70, 129, 1)]
    outs = []
    for graphs in (True, False):
        eng = G.engine(m, pages=40, block_size=64, use_cuda_graphs=graphs)
        outs.append([r.out_tokens for r in eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))])
        assert bool(eng._graphs) == graphs
    assert outs[0] == outs[1]
