"""Gadarax (layer-list models: latent attention, retention, dynamic tanh, looped layers) on the CPU: every mechanism and the whole
engine against the float64 statement in ``gadarax_oracle``."""

import io
import json
import sys

import gadarax_cases as G
import gadarax_oracle as O
import pytest
import torch

from rl_b200.engine.engine import SamplingParams, _NativeScheduler, _PyScheduler
from rl_b200.models.config import ModelConfig, preset, rotary_table
from rl_b200.models.hf_io import load_pretrained, save_pretrained
from rl_b200.models.mixers import DynamicTanh, LatentAttentionMixer, RetentionMixer, rotate_pairs
from rl_b200.models.transformer import PackedBatch, build_model
from rl_b200.ops import lib as L
from rl_b200.ops import mixer_ops as X

TOL = 2e-5


class Cfg:
    rms_norm_eps = 1e-5


@pytest.fixture(scope="module", params=sorted(G.CASES))
def case(request, tmp_path_factory):
    cfg = G.CASES[request.param]
    w = G.weights(cfg, seed=7)
    return cfg, w, G.load(cfg, w, tmp_path_factory.mktemp(request.param))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("rot", [dict(dims=8, base=10000.0), dict(dims=2, base=500.0), dict(dims=16, base=1e6, scaling=dict(G.YARN)),
                                 dict(dims=16, base=1e4, scaling=dict(factor=8.0, original=1 << 22, fast=32.0, slow=1.0)),    # ramp reaches past the pairs
                                 dict(dims=8, base=1e4, scaling=dict(factor=2.0, original=6, fast=64.0, slow=32.0))])         # every pair is slowed
def test_rotary_table(rot):
    f, gain = rotary_table(rot)
    want, m = O.frequencies(rot)
    assert gain == pytest.approx(m, rel=1e-12)
    assert torch.allclose(f.double(), torch.tensor(want, dtype=torch.float64), rtol=1e-7)


@pytest.mark.parametrize("interleaved", [True, False])
@pytest.mark.parametrize("dims", [0, 2, 6, 10])
def test_rotation(interleaved, dims):
    rot = dict(dims=dims, base=100.0, scaling=dict(G.YARN)) if dims else dict(dims=0, base=100.0)
    x = torch.randn(9, 3, 10, dtype=torch.float64)
    f, gain = rotary_table(rot)
    got = rotate_pairs(x, torch.arange(70, 79), f, gain, interleaved)
    assert torch.allclose(got.double(), O.rotate(x, rot, 70, interleaved), atol=1e-5)


def test_dynamic_tanh_and_epilogues():
    torch.manual_seed(0)
    n = DynamicTanh(24, torch.float32, "cpu")
    with torch.no_grad():
        n.weight.normal_(), n.bias.normal_(), n.alpha.fill_(-0.7)
        x, e, a, w, st = torch.randn(5, 24), torch.randn(5, 24), torch.randn(5, 16), torch.randn(24, 16), torch.randn(24)
        ref = O.dyt(x.double(), n.weight.double(), n.bias.double(), n.alpha.double())
        assert torch.allclose(n(x).double(), ref, atol=1e-6)
        want = x.double() + a.double() @ w.double().T + e + st
        h = X.out_proj_(x, a, w, e, st, n)
        assert torch.allclose(x.double(), want, atol=1e-5)
        assert torch.allclose(h.double(), O.dyt(want, n.weight.double(), n.bias.double(), n.alpha.double()), atol=1e-5)
        p = X.in_proj(a, w, 8)
        ref = a.double() @ w.double().T
        ref[:, 8:] = torch.relu(ref[:, 8:]) ** 2
        assert torch.allclose(p.double(), ref, atol=1e-5)


@pytest.mark.parametrize("entry", [G.latent(scaling=G.YARN), G.latent(heads=1, dim=5, rot_dim=6, vdim=7, kv_rank=9), G.latent(heads=2, dim=8, rot_dim=4, vdim=8, kv_rank=8, scale=2.0)])
def test_latent_attention_alone(entry):
    cfg = G.config([entry])
    w = {k: v.double() for k, v in O.below(G.weights(cfg, 3), "l0.mix.").items()}
    m = LatentAttentionMixer(entry["mixer"], Cfg, torch.float32, "cpu")
    h = torch.randn(23, cfg["width"], dtype=torch.float64)
    with torch.no_grad():
        W = torch.zeros(m.in_width, cfg["width"])
        for leaf, r, n in m.in_rows():
            W[r : r + n] = w[leaf].float()
        m.kv_norm.copy_(w["dkv.norm"])
        m.kv_up.copy_(torch.cat([w["uk"], w["uv"]]))
        y = m.sequence(h.float() @ W.T, torch.arange(23), torch.tensor([0, 23])).double()
    assert torch.allclose(y @ w["o"].T, O.latent_attention(w, h, entry["mixer"], 1e-5), atol=2e-5)


@pytest.mark.parametrize("entry", [G.retention(), G.retention(heads=2, dim=6, vdim=10, rot_dims=2, decay=[1.0, 0.25])])
def test_retention_alone_and_its_state(entry):
    cfg = G.config([entry])
    w = {k: v.double() for k, v in O.below(G.weights(cfg, 3), "l0.mix.").items()}
    m = RetentionMixer(entry["mixer"], Cfg, torch.float32, "cpu")
    T = 150
    h = torch.randn(T, cfg["width"], dtype=torch.float64)
    W = torch.zeros(m.in_width, cfg["width"])
    for leaf, r, n in m.in_rows():
        W[r : r + n] = w[leaf].float()
    p = h.float() @ W.T
    want, S = O.retention(w, h, entry["mixer"], 1e-5)
    y = m.sequence(p, torch.arange(T), torch.tensor([0, T])).double()
    assert torch.allclose(y @ w["o"].T, want, atol=3e-5)
    q, k, v = m.qkv(p, torch.arange(T))
    for chunk in (1, 2, 64, 200):
        _, s = m.scan(q, k, v, torch.zeros(m.heads, m.dim, m.vdim), chunk)
        assert torch.allclose(s.double(), S, atol=1e-4)


def test_config_round_trip_and_checks(tmp_path):
    cfg = G.CASES["loop"]
    c = ModelConfig.from_hf_dict(cfg)
    assert c.is_mixer and c.is_recurrent and not ModelConfig.from_hf_dict(G.CASES["attention_only"]).is_recurrent
    assert c.layer_runs == O.run_order(cfg) and len(c.layer_runs) == 8
    back = ModelConfig.from_hf_dict(json.loads(json.dumps(c.to_hf_dict())))
    assert back == c
    w = G.weights(cfg, 1)
    m = G.load(cfg, w, tmp_path / "a")
    assert c.num_parameters() == sum(v.numel() for v in w.values())
    save_pretrained(m, str(tmp_path / "b"), dtype=torch.bfloat16)
    from safetensors.torch import load_file

    again = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(again) == set(w) and all(torch.equal(again[k], w[k]) for k in w)
    for bad in ({"type": "nothing"}, {"mixer": {"heads": 2}}):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[dict(cfg["layers"][0], **bad)], loop=None))
    with pytest.raises(ValueError):
        ModelConfig.from_hf_dict(dict(cfg, loop={"start": 3, "stop": 2, "times": 1}))
    with pytest.raises(KeyError):
        from safetensors.torch import save_file

        save_file({k: v for k, v in w.items() if k != "l1.mix.g"}, str(tmp_path / "a" / "model.safetensors"))
        load_pretrained(str(tmp_path / "a"))


def test_trains(case):
    cfg, w, model = case
    toks = G.tokens(cfg, 30)
    ids = torch.tensor(toks)
    b = PackedBatch(ids, torch.cat([torch.arange(12), torch.arange(18)]).int(), torch.tensor([0, 12, 30], dtype=torch.int32), 18)
    z = model.logits(b)
    want = torch.cat([G.oracle(cfg, w, toks[:12]), G.oracle(cfg, w, toks[12:])])
    assert G.gap(z.detach(), want) < TOL
    lp, _ = model.next_token_logprobs(b)
    lp.sum().backward()
    named = dict(model.named_parameters())
    assert all(p.grad is not None and torch.isfinite(p.grad).all() for p in named.values())
    model.zero_grad(set_to_none=True)


def test_random_init_and_presets():
    m = build_model(preset("tiny-gadarax"), seed=3, dtype=torch.float32)
    assert (m.layers[0].norm.weight == 1).all() and m.layers[0].in_proj.std() > 0.01
    assert build_model(preset("tiny-gadarax"), seed=3, dtype=torch.float32).layers[1].out_proj.equal(m.layers[1].out_proj)
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-gadarax"), pp_size=2)


def test_worker_trains_and_generates():
    """The policy worker around the model: rollout log-probabilities equal the trainer's, and a few steps lower the loss."""
    from rl_b200.algorithms.loss.loss_functions import NLLLossFn
    from rl_b200.distributed.batched_data_dict import BatchedDataDict
    from rl_b200.policy.worker import PolicyWorker
    from rl_b200.utils.flops import model_flops

    mc = preset("tiny-gadarax")
    assert model_flops(mc, 20) > 0
    p = PolicyWorker(dict(precision="float32", train_global_batch_size=4, train_micro_batch_size=2, max_total_sequence_length=64,
                          optimizer=dict(name="torch.optim.AdamW", kwargs=dict(lr=1e-3)),
                          generation=dict(max_new_tokens=8, stop_token_ids=[], kv_cache_tokens=1024, block_size=16, max_running=4)),
                     model_cfg=mc, device="cpu", init_reference_model=False)
    recs = p.build_generation().engine.generate([G.tokens({"vocab": 264}, 12, s) for s in range(4)], SamplingParams(max_new_tokens=8, seed=1))
    ids = torch.tensor([r.prompt + r.out_tokens for r in recs])
    data = BatchedDataDict(input_ids=ids, input_lengths=torch.full((4,), 20), token_mask=torch.ones(4, 20), sample_mask=torch.ones(4))
    lp = p.get_logprobs(data)["logprobs"][:, 12:]
    assert torch.allclose(lp, torch.tensor([r.out_logprobs for r in recs]), atol=1e-5)
    losses = [float(p.train(data, NLLLossFn(), gbs=4, mbs=2)["loss"]) for _ in range(3)]
    assert losses[2] < losses[0]


# ------------------------------------------------------------------------------------------------ engine
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3], [16], [17, 2, 33, 1], [50, 1]])
def test_portions_equal_the_oracle(case, cuts):
    cfg, w, model = case
    toks = G.tokens(cfg, 70)
    eng = G.engine(model)
    assert G.gap(G.run_cut(eng, "a", toks, cuts), G.oracle(cfg, w, toks)) < TOL
    assert eng.sched.num_free_blocks == 24


def test_mixed_batches_and_reused_pages(case):
    """More requests than pages and state slots hold at once, in random batches; each equals itself alone."""
    cfg, w, model = case
    seqs = {f"r{i}": G.tokens(cfg, n, seed=i) for i, n in enumerate([60, 1, 33, 17, 48, 2, 80, 16])}
    steps = G.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = G.engine(model, pages=G.live_pages(steps, 16))
    got = G.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert G.gap(got[r], G.oracle(cfg, w, t)) < TOL, r
    assert not eng._step_ids and eng.sched.num_free_blocks == eng.num_blocks


def test_step_limits(case):
    cfg, _, model = case
    eng = G.engine(model, pages=3, requests=2)
    eng.step([("a", [1, 2, 3], []), ("b", [4], [])])
    with pytest.raises(RuntimeError, match="live requests"):
        eng.step([("c", [1], [])])
    with pytest.raises(RuntimeError, match="no room"):
        eng.step([("a", [1] * 40, [])])
    with pytest.raises(ValueError, match="two entries"):
        eng.step([("a", [1], []), ("a", [1], [])])
    eng.step([("a", [5], [0])], ["a", "b"])
    assert eng.step([("c", [1] * 40, [39])], ["c"])[0].shape == (1, cfg["vocab"])


def greedy(cfg, w, prompt, n):
    out = list(prompt)
    for _ in range(n):
        out.append(int(G.oracle(cfg, w, out)[-1].argmax()))
    return out[len(prompt) :]


def test_greedy_generation(case):
    """Through the engine's own entry point and scheduler: unequal prompts, fewer running slots than requests, chunked prefill."""
    cfg, w, model = case
    prompts = [G.tokens(cfg, n, seed=n) for n in (1, 5, 16, 17, 40, 5)]
    prompts[5] = list(prompts[1])      # an equal prompt (shared where the model has no state)
    eng = G.engine(model, requests=3, max_prefill_tokens=24)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=9))
    for p, r in zip(prompts, recs):
        assert r.out_tokens == greedy(cfg, w, p, 9)
    again = eng.generate(prompts[::-1], SamplingParams(greedy=True, max_new_tokens=9))
    assert [r.out_tokens for r in again[::-1]] == [r.out_tokens for r in recs]


def test_preemption_rebuilds_the_state(case):
    cfg, w, model = case
    prompts = [G.tokens(cfg, 20, seed=s) for s in range(3)]
    eng = G.engine(model, pages=6, requests=3)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))
    assert eng.sched.num_preemptions > 0
    big = G.engine(model, pages=40, requests=3).generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))
    assert [r.out_tokens for r in recs] == [r.out_tokens for r in big]


@pytest.mark.parametrize("far", [0, 1, 15, 16, 17, 31, 32, 62, 63])
@pytest.mark.parametrize("n", [1, 2, 20, 64])
def test_one_key_far_away(far, n):
    """One key holds all the weight of every query that sees it: at the first tokens, at page borders, at the query itself."""
    T, bs = 64, 16
    m, p, b, cache, want = standout_case(T, bs, far, n)
    X.latent_attention_(p, m, b, cache)
    got = p[:, m.mix_off : m.mix_off + m.heads * m.vdim].float()
    rows = [i for i in range(n) if T - n + i >= far]
    assert torch.allclose(got[rows], want[rows], atol=1e-4)
    hidden = [i for i in range(n) if T - n + i < far]       # queries before it must not see it
    assert not hidden or (got[hidden] - want[hidden]).abs().max() > 1e-2


def standout_case(T, bs, far, n, device="cpu", dtype=torch.float32, heads=2, dim=16, rot_dim=8, vdim=8, rank=24):
    """A batch of ``n`` new tokens behind ``T - n`` cached ones whose pages are scattered; every query scores key ``far`` far above all
    others. Returns (mixer, projected rows, batch, cache, outputs if that key alone counted)."""
    g = torch.Generator().manual_seed(far * 100 + n)
    m = LatentAttentionMixer(G.latent(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank)["mixer"], Cfg, dtype, device)
    H, R = m.heads, m.rank
    lat = torch.randn(T, R, generator=g) * 0.5
    lat[:, 0] = -3.0
    lat[far, 0] = 3.0
    lat = lat / lat.pow(2).mean(-1, keepdim=True).sqrt()
    with torch.no_grad():
        uk = torch.zeros(H, m.dim, R)
        uk[:, 0, 0] = 1.0
        m.kv_up.copy_(torch.cat([uk.reshape(-1, R), torch.randn(H * m.vdim, R, generator=g)]).to(m.kv_up.dtype))
    pages = -(-T // bs)
    order = torch.randperm(pages + 3, generator=g)[:pages]
    cache = torch.randn(pages + 3, bs, m.latent_width, generator=g).to(device, dtype)
    cache[..., R + m.rot_dim :] = 0
    slot = order[torch.arange(T) // bs] * bs + torch.arange(T) % bs
    flat = cache.view(-1, m.latent_width)
    old = slot[: T - n].to(device)
    flat[old, :R] = lat[: T - n].to(device, dtype)
    flat[old, R:] = 0
    p = torch.zeros(n, m.in_width)
    q = p[:, : H * m.qdim].view(n, H, m.qdim)
    q[:, :, 0] = 40.0
    p[:, m.lat_off : m.lat_off + R] = lat[T - n :]
    p = p.to(device, dtype)                              # gate 0: sigmoid 1/2
    pos = torch.arange(T - n, T, dtype=torch.int32)
    bt = torch.zeros(1, pages + 1, dtype=torch.int32)
    bt[0, :pages] = order
    b = X.TokenBatch(ids=None, positions=pos.to(device), slots=slot[T - n :].to(device), n_single=int(n == 1), n_paged=n,
                     block_table=bt.expand(n, -1).contiguous().to(device), seq_lens=(pos + 1).to(device), max_ctx=T)
    if device != "cpu" and n > X.PAGED_PORTION and X.portion_tiles(m, dtype):
        cu = torch.tensor([[0, n], [0, T]], dtype=torch.int32, device=device)
        b.n_paged, b.block_table, b.seq_lens = 0, b.block_table[:0], b.seq_lens[:0]
        b.cu_q, b.cu_ctx, b.q_tiles, b.ctx_slots = cu[0], cu[1], -(-n // 128), slot.to(device)
    c = lat[far] if far < T - n else lat[far] / (lat[far].pow(2).mean() + m.eps).sqrt()
    y = (m.kv_up[H * m.dim :].float().cpu() @ c) * 0.5
    return m, p, b, cache, y.expand(n, -1)


def test_scheduler_stepped_sequences():
    scheds = [_PyScheduler(6, 4, 4, 0)] + ([_NativeScheduler(6, 4, 4, 0)] if L.available() else [])
    for s in scheds:
        assert s.open(7) == 0 and s.open(7) == -1
        assert s.extend(7, 5) == 0 and s.extend(7, 1) == 5 and s.extend(9, 1) == -1
        assert s.num_free_blocks == 4 and s.extend(7, 40) == -2 and s.num_free_blocks == 4
        assert s.slots(7, 0, 6).numel() == 6
        assert s.add(1, 4, 2, -1) == 0                       # scheduled requests live beside stepped ones
        pf, sh, dc, cp = s.schedule()
        assert pf == [1] and not dc
        assert s.close(7) == 0 and s.close(7) == -1 and s.num_free_blocks == 4


def test_trace_runner(tmp_path, monkeypatch, capsys):
    from rl_b200.tools.trace_run import main

    cfg = G.CASES["loop"]
    w = G.weights(cfg, 2)
    path = G.save(cfg, w, tmp_path / "m")
    a, b = G.tokens(cfg, 21, 1), G.tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[20:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert main(["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]) == 0
    assert [l for l in capsys.readouterr().out.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    za, zb = G.oracle(cfg, w, a), G.oracle(cfg, w, b)

    def read(n):
        return torch.frombuffer(bytearray((tmp_path / "o" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    assert G.gap(read(0), torch.stack([za[0], za[19], zb[0]])) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    assert G.gap(read(2), torch.stack([zb[8], za[20]])) < TOL


@pytest.mark.parametrize("family", ["llama", "nemotron_h"])
def test_step_serves_other_families(family):
    """The same step function drives the other model families (whole prompts, portions and single tokens in one batch)."""
    mc = preset("tiny-nemotron-h") if family == "nemotron_h" else ModelConfig(
        vocab_size=97, hidden_size=32, intermediate_size=64, num_hidden_layers=2, num_attention_heads=4, num_key_value_heads=2, head_dim=8)
    m = build_model(mc, seed=1, dtype=torch.float32)
    eng = G.engine(m, pages=12)
    seqs = {"a": G.tokens({"vocab": mc.vocab_size}, 30, 1), "b": G.tokens({"vocab": mc.vocab_size}, 23, 2)}
    got = G.run_schedule(eng, [{"a": 17}, {"a": 1, "b": 9}, {"b": 1, "a": 2}, {"a": 10, "b": 13}], seqs)
    for r, t in seqs.items():
        n = len(t)
        z = m.logits(PackedBatch(torch.tensor(t), torch.arange(n).int(), torch.tensor([0, n], dtype=torch.int32), n)).detach()
        assert (got[r] - z).abs().max() < 1e-3 * z.abs().max()
