"""Redarax (post-norm layer-list models: grouped attention, Mamba-2, gated delta rule, clamped experts, token inputs) on the CPU: every
mechanism and the whole engine against the float64 statement in ``redarax_oracle``."""

import io
import json
import sys

import pytest
import redarax_cases as R
import redarax_oracle as O
import torch

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import ModelConfig, preset
from rl_b200.models.hf_io import load_pretrained, save_pretrained
from rl_b200.models.mixers import DeltaMixer, GroupedAttentionMixer, Mamba2LayerMixer
from rl_b200.models.gated import GatedExperts, GatedUnit, clamped_glu
from rl_b200.models.transformer import PackedBatch, build_model
from rl_b200.ops import layer_ops as Y
from rl_b200.ops import mixer_ops as X
from rl_b200.ops import sequence_ops as S

TOL = 2e-4        # (fp32 against float64; the small random models amplify roundings)
F64 = torch.float64


class Cfg:
    rms_norm_eps = 1e-5
    hidden_size = 56


@pytest.fixture(scope="module", params=sorted(R.CASES))
def case(request, tmp_path_factory):
    cfg = R.CASES[request.param]
    w = R.weights(cfg, seed=7)
    return cfg, w, R.load(cfg, w, tmp_path_factory.mktemp(request.param))


def alone(entry, seed=3):
    w = {k: v.to(F64) for k, v in O.below(R.weights(R.config([(entry, None)]), seed), "l0.mix.").items()}
    cls = {"attention": GroupedAttentionMixer, "mamba2": Mamba2LayerMixer, "delta": DeltaMixer}[entry["type"]]
    return w, R.module_weights(cls(entry["mixer"], Cfg, torch.float32, "cpu"), w)


def project(m, h):
    p = h.float() @ m.in_proj.t()
    return (p if m.in_bias is None else p + m.in_bias).detach()


def out(m, y):
    y = y.double() @ m.out_proj[:, : y.shape[1]].double().t()
    return (y if m.out_bias is None else y + m.out_bias.double()).detach()


# ------------------------------------------------------------------------------------------------ mechanisms
MIXERS = [R.attention(), R.attention(heads=3, kv_heads=3, dim=5, vdim=9, rot_dims=4, scale=1.0), R.attention(heads=8, kv_heads=2, dim=8, vdim=8, rot_dims=0),
          R.mamba2(), R.mamba2(heads=2, vdim=5, state=3, groups=2, norm_groups=1, conv=1), R.mamba2(heads=4, vdim=6, groups=1, norm_groups=4, conv=5),
          R.delta(), R.delta(heads=1, kv_heads=1, dim=3, vdim=4, conv=1), R.delta(heads=6, kv_heads=3, dim=16, vdim=8, conv=6)]


@pytest.mark.parametrize("entry", MIXERS)
def test_mixer_alone(entry):
    w, m = alone(entry)
    h = torch.randn(80, 56, dtype=F64)
    y = m.sequence(project(m, h), torch.arange(80), torch.tensor([0, 80]))
    assert torch.allclose(out(m, y), O.MIXERS[entry["type"]](w, h, entry["mixer"], 1e-5), atol=3e-5)


@pytest.mark.parametrize("entry", [e for e in MIXERS if e["type"] != "attention"])
@pytest.mark.parametrize("cuts", [[80], [1] * 80, [2] * 40, [3, 64, 1, 1, 11], [65, 15]])
def test_recurrent_state_is_carried(entry, cuts):
    """Pieces through the operator: ring and state rows carry what a later piece needs; a piece at position 0 forgets what they held."""
    w, m = alone(entry)
    h = torch.randn(80, 56, dtype=F64)
    want = O.MIXERS[entry["type"]](w, h, entry["mixer"], 1e-5)
    ring, state = torch.randn(3, m.taps, m.channels), torch.randn(3, m.heads, m.dim, m.vdim)
    keep = state[0].clone(), ring[0].clone()
    got, at = [], 0
    for n in cuts:
        b = X.TokenBatch(ids=None, positions=torch.arange(at, at + n, dtype=torch.int32), slots=None, n_single=int(n == 1), n_paged=0, block_table=None,
                         seq_lens=None, state_rows=torch.tensor([2]), cu=None if n == 1 else torch.tensor([0, n]))
        got.append(out(m, S.recurrent(project(m, h[at : at + n]), m, b, ring, state)[:, : m.heads * m.vdim]))
        at += n
    assert torch.allclose(torch.cat(got), want, atol=3e-5)
    assert torch.equal(state[0], keep[0]) and torch.equal(ring[0], keep[1])


def test_delta_rule_corrects_what_it_stores():
    """Two writes under one key: the second replaces the first (beta 1, no decay), which a plain linear-attention state would sum."""
    m = DeltaMixer(R.delta(heads=1, kv_heads=1, dim=4, vdim=3, conv=1)["mixer"], Cfg, torch.float32, "cpu")
    with torch.no_grad():
        m.A_log.fill_(-30.0)
    u = torch.zeros(3, m.channels)
    u[:, :4] = u[:, 4:8] = torch.tensor([1.0, 2.0, -1.0, 0.5])
    u[0, 8:], u[1, 8:], u[2, 8:] = torch.tensor([5.0, 5.0, 5.0]), torch.tensor([1.0, -2.0, 3.0]), torch.tensor([1.0, -2.0, 3.0])
    p = torch.zeros(3, m.in_width)
    p[:, m.b_off] = 40.0
    o, _ = m.scan(u, p, torch.zeros(1, 4, 3))
    assert torch.allclose(o[1, 0] * 2, torch.tensor([1.0, -2.0, 3.0]), atol=1e-5) and torch.allclose(o[0, 0] * 2, torch.tensor([5.0] * 3), atol=1e-5)


def test_clamped_unit_and_its_limits():
    p = torch.tensor([[9.0, 0.5, -9.0, 0.5, 0.3, 9.0, 0.3, -9.0, 0.2, -0.4]], dtype=F64)
    got = Y.clamped_glu_ref(p.float(), 1.5)
    g, u = p[:, 0::2].clamp(max=1.5), p[:, 1::2].clamp(-1.5, 1.5)
    want = g / (1 + torch.exp(-1.702 * g)) * (u + 1)
    assert torch.allclose(got.double(), want, atol=1e-6) and torch.allclose(clamped_glu(p.float(), 1.5).double(), want, atol=1e-6)
    for spec in (R.dense(), R.dense(ff=9, limit=0.3)):
        w = {k: v.to(F64) for k, v in O.below(R.weights(R.config([(R.delta(), spec)]), 1), "l0.mlp.").items()}
        m = R.module_weights(GatedUnit(spec, Cfg, torch.float32, "cpu"), w)
        h = torch.randn(30, 56, dtype=F64)
        assert torch.allclose(m(h.float()).double(), O.clamped_glu(w, h, spec["limit"]), atol=2e-5)
        assert torch.allclose(Y.linear(Y.linear(h.float(), m.gate_up, glu=m.limit), m.down).double(), O.clamped_glu(w, h, spec["limit"]), atol=2e-5)


@pytest.mark.parametrize("spec", [R.moe(), R.moe(experts=5, top=2, groups=None), R.moe(experts=6, top=6, groups=(1, 1)), R.moe(experts=12, top=4, groups=(3, 2)),
                                  R.moe(experts=6, top=2, groups=(6, 3)), R.moe(experts=8, top=2, groups=(2, 1))])
def test_experts_alone(spec):
    w = {k: v.to(F64) for k, v in O.below(R.weights(R.config([(R.delta(), spec)]), 5), "l0.mlp.").items()}
    m = R.module_weights(GatedExperts(spec, Cfg, torch.float32, "cpu"), w)
    h = torch.randn(60, 56, dtype=F64)
    want = O.experts(w, h, spec)
    assert torch.allclose(m(h.float()).double(), want, atol=3e-5)
    assert torch.allclose(Y.gated_experts(h.float(), m)[0].double(), want, atol=3e-5)


def test_router_masks_groups_with_minus_infinity():
    """All choice scores negative: experts of dropped groups must not win over eligible ones (a mask of 0 would let them)."""
    spec = R.moe(experts=6, top=2, groups=(3, 1))
    m = GatedExperts(spec, Cfg, torch.float32, "cpu")
    m.correction.copy_(torch.tensor([-3.0, -3.0, -2.0, -2.0, -4.0, -1.9]))
    wt, idx = m.choose(torch.zeros(1, 6))
    assert sorted(idx[0].tolist()) == [2, 3] and torch.allclose(wt, torch.full((1, 2), 0.5))
    assert [e for e, _ in O.route({"router": torch.zeros(6, 4, dtype=F64), "correction": m.correction.double()}, torch.zeros(1, 4, dtype=F64), spec["router"])[0]] == [2, 3]


def test_join_norms_and_cap():
    torch.manual_seed(0)
    x, y, w, nw = torch.randn(5, 24), torch.randn(5, 24) * 1e-2, torch.randn(24), torch.randn(24)
    want = x.double() + 0.7 * O.rms(y.double(), 1e-3) * w.double()
    x1 = x.clone()
    assert torch.allclose(Y.add_normed_(x1, y, w, 0.7, 1e-3).double(), want, atol=1e-5) and torch.allclose(x1.double(), want, atol=1e-5)
    x1 = x.clone()
    assert torch.allclose(Y.add_normed_(x1, y, w, 0.7, 1e-3, nw).double(), O.rms(want, 1e-3) * nw.double(), atol=1e-5)
    g = torch.randn(4, 30)
    z = g.clone()
    Y.group_norm_(z, w[:24], 3, 1e-3)
    assert torch.allclose(z[:, :24].double(), O.rms(g[:, :24].double().view(4, 3, 8), 1e-3).view(4, 24) * w.double(), atol=1e-5) and torch.equal(z[:, 24:], g[:, 24:])
    h, v = torch.randn(3, 24), torch.randn(40, 24)
    assert torch.allclose(Y.capped_logits(h, v, 2.0, 3.0).double(), 3 * torch.tanh(h.double() @ v.double().t() * 2 / 3), atol=1e-5)


def test_config_round_trip_and_checks(tmp_path):
    cfg = R.CASES["all"]
    c = ModelConfig.from_hf_dict(cfg)
    assert c.is_mixer and c.is_recurrent and c.caps_logits and not ModelConfig.from_hf_dict(R.CASES["attention_only"]).is_recurrent
    for name, k in R.CASES.items():
        c = ModelConfig.from_hf_dict(k)
        assert ModelConfig.from_hf_dict(json.loads(json.dumps(c.to_hf_dict()))) == c
        assert c.num_parameters() == sum(v.numel() for v in R.weights(k).values()), name
    w = R.weights(cfg, 1)
    m = R.load(cfg, w, tmp_path / "a")
    save_pretrained(m, str(tmp_path / "b"), dtype=torch.bfloat16)
    from safetensors.torch import load_file, save_file

    again = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(again) == set(w) and all(torch.equal(again[k], w[k]) for k in w)
    l0 = cfg["layers"][0]
    for bad in ({"type": "retention"}, {"mixer": {"heads": 2}}, {"mixer": dict(l0["mixer"], groups=4)}, {"mixer": dict(l0["mixer"], norm_groups=5)},
                {"mlp": {"kind": "sparse", "ff": 3}}, {"mlp": R.moe(experts=8, top=5, groups=(4, 2))}):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[dict(l0, **bad)]))
    with pytest.raises(KeyError):
        save_file({k: v for k, v in w.items() if k != "l1.mix.g"}, str(tmp_path / "a" / "model.safetensors"))
        load_pretrained(str(tmp_path / "a"))


def test_trains(case):
    cfg, w, model = case
    toks = R.tokens(cfg, 30)
    b = PackedBatch(torch.tensor(toks), torch.cat([torch.arange(12), torch.arange(18)]).int(), torch.tensor([0, 12, 30], dtype=torch.int32), 18)
    z = model.logits(b)
    want = torch.cat([R.oracle(cfg, w, toks[:12]), R.oracle(cfg, w, toks[12:])])
    assert R.gap(z.detach(), want) < TOL
    lp, ent = model.next_token_logprobs(b, want_entropy=True)
    ref = torch.log_softmax(want, -1)
    assert torch.allclose(lp[1:12].double(), ref[:11].gather(-1, torch.tensor(toks[1:12])[:, None])[:, 0], atol=1e-3)
    assert torch.allclose(ent[1:12].double(), -(ref[:11].exp() * ref[:11]).sum(-1), atol=1e-3)
    lp.sum().backward()
    named = dict(model.named_parameters())
    assert all(p.grad is not None and torch.isfinite(p.grad).all() for p in named.values())
    model.zero_grad(set_to_none=True)


def test_worker_trains_and_generates():
    from rl_b200.algorithms.loss.loss_functions import NLLLossFn
    from rl_b200.distributed.batched_data_dict import BatchedDataDict
    from rl_b200.policy.worker import PolicyWorker
    from rl_b200.utils.flops import model_flops

    mc = preset("tiny-redarax")
    assert model_flops(mc, 20) > 0
    p = PolicyWorker(dict(precision="float32", train_global_batch_size=4, train_micro_batch_size=2, max_total_sequence_length=64,
                          optimizer=dict(name="torch.optim.AdamW", kwargs=dict(lr=1e-3)),
                          generation=dict(max_new_tokens=8, stop_token_ids=[], kv_cache_tokens=1024, block_size=16, max_running=4)),
                     model_cfg=mc, device="cpu", init_reference_model=False)
    recs = p.build_generation().engine.generate([R.tokens({"vocab": 264}, 12, s) for s in range(4)], SamplingParams(max_new_tokens=8, seed=1))
    ids = torch.tensor([r.prompt + r.out_tokens for r in recs])
    data = BatchedDataDict(input_ids=ids, input_lengths=torch.full((4,), 20), token_mask=torch.ones(4, 20), sample_mask=torch.ones(4))
    lp = p.get_logprobs(data)["logprobs"][:, 12:]
    assert torch.allclose(lp, torch.tensor([r.out_logprobs for r in recs]), atol=1e-4)
    losses = [float(p.train(data, NLLLossFn(), gbs=4, mbs=2)["loss"]) for _ in range(3)]
    assert losses[2] < losses[0]


def test_random_init():
    m = build_model(preset("tiny-redarax"), seed=3, dtype=torch.float32)
    assert (m.layers[0].norm1 == 1).all() and m.layers[0].mixer.in_proj.std() > 0.01 and (m.layers[0].mixer.dt_bias < 0).all()
    assert build_model(preset("tiny-redarax"), seed=3, dtype=torch.float32).layers[1].ff.down.equal(m.layers[1].ff.down)
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-redarax"), pp_size=2)


# ------------------------------------------------------------------------------------------------ engine
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3], [16], [17, 2, 33, 1], [50, 1]])
def test_portions_equal_the_oracle(case, cuts):
    cfg, w, model = case
    toks = R.tokens(cfg, 70)
    eng = R.engine(model)
    assert R.gap(R.run_cut(eng, "a", toks, cuts), R.oracle(cfg, w, toks)) < TOL
    assert eng.sched.num_free_blocks == 24


def test_mixed_batches_and_reused_pages(case):
    cfg, w, model = case
    seqs = {f"r{i}": R.tokens(cfg, n, seed=i) for i, n in enumerate([60, 1, 33, 17, 48, 2, 80, 16])}
    steps = R.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = R.engine(model, pages=R.live_pages(steps, 16))
    got = R.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert R.gap(got[r], R.oracle(cfg, w, t)) < TOL, r
    assert not eng._step_ids and eng.sched.num_free_blocks == eng.num_blocks


def greedy(cfg, w, prompt, n):
    o = list(prompt)
    for _ in range(n):
        o.append(int(R.oracle(cfg, w, o)[-1].argmax()))
    return o[len(prompt) :]


def test_greedy_generation(case):
    cfg, w, model = case
    prompts = [R.tokens(cfg, n, seed=n) for n in (1, 5, 16, 17, 40, 5)]
    prompts[5] = list(prompts[1])
    eng = R.engine(model, requests=3, max_prefill_tokens=24)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=9))
    for p, r in zip(prompts, recs):
        assert r.out_tokens == greedy(cfg, w, p, 9)
    again = eng.generate(prompts[::-1], SamplingParams(greedy=True, max_new_tokens=9))
    assert [r.out_tokens for r in again[::-1]] == [r.out_tokens for r in recs]


def test_preemption_rebuilds_the_state(case):
    cfg, w, model = case
    prompts = [R.tokens(cfg, 20, seed=s) for s in range(3)]
    eng = R.engine(model, pages=6, requests=3)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))
    assert eng.sched.num_preemptions > 0
    big = R.engine(model, pages=40, requests=3).generate(prompts, SamplingParams(greedy=True, max_new_tokens=40))
    assert [r.out_tokens for r in recs] == [r.out_tokens for r in big]


def standout_case(T, bs, far, n, device="cpu", dtype=torch.float32, heads=4, kv_heads=2, dim=16, vdim=8, rot_dims=0):
    """``n`` new tokens behind ``T - n`` cached ones in scattered pages; every query scores key ``far`` far above all others. Returns
    (mixer, projected rows, batch, key cache, value cache, outputs if that key alone counted)."""
    g = torch.Generator().manual_seed(far * 100 + n)
    m = GroupedAttentionMixer(R.attention(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot_dims=rot_dims, scale=2.0)["mixer"], Cfg, dtype, device)
    k = torch.full((T, kv_heads, dim), 0.1)
    k[:, :, 0] = -1.0
    k[far, :, 0] = 1.0
    k = k / k.pow(2).mean(-1, keepdim=True).sqrt()
    v = torch.randn(T, kv_heads, vdim, generator=g)
    pages = -(-T // bs)
    order = torch.randperm(pages + 3, generator=g)[:pages]
    kc, vc = (torch.randn(pages + 3, kv_heads, bs, w, generator=g) for w in (dim, vdim))
    t = torch.arange(T)
    slot = order[t // bs] * bs + t % bs
    kc[slot[: T - n] // bs, :, slot[: T - n] % bs], vc[slot[: T - n] // bs, :, slot[: T - n] % bs] = k[: T - n], v[: T - n]
    p = torch.zeros(n, m.in_width)
    p[:, m.q_off : m.q_off + heads * dim].view(n, heads, dim)[:, :, 0] = 30.0
    p[:, m.k_off : m.k_off + kv_heads * dim] = k[T - n :].reshape(n, -1)
    p[:, m.v_off : m.v_off + kv_heads * vdim] = v[T - n :].reshape(n, -1)
    pos = torch.arange(T - n, T, dtype=torch.int32)
    bt = torch.zeros(1, pages + 1, dtype=torch.int32)
    bt[0, :pages] = order
    b = X.TokenBatch(ids=None, positions=pos.to(device), slots=slot[T - n :].to(device), n_single=int(n == 1), n_paged=n,
                     block_table=bt.expand(n, -1).contiguous().to(device), seq_lens=(pos + 1).to(device), max_ctx=T)
    if device != "cpu" and n > X.PAGED_PORTION and S.portion_tiles(m, dtype):
        cu = torch.tensor([[0, n], [0, T]], dtype=torch.int32, device=device)
        b.n_paged, b.block_table, b.seq_lens, b.whole = 0, b.block_table[:0], b.seq_lens[:0], n == T
        b.cu_q, b.cu_ctx, b.q_tiles, b.ctx_slots = cu[0], cu[1], -(-n // 128), slot.to(device)
    want = v[far].repeat_interleave(heads // kv_heads, 0).reshape(-1)
    return m, p.to(device, dtype), b, kc.to(device, dtype), vc.to(device, dtype), want.expand(n, -1)


@pytest.mark.parametrize("far", [0, 1, 15, 16, 17, 31, 32, 62, 63])
@pytest.mark.parametrize("n", [1, 2, 20, 64])
def test_one_key_far_away(far, n):
    T, bs = 64, 16
    m, p, b, kc, vc, want = standout_case(T, bs, far, n)
    with torch.no_grad():
        got = S.attention(p, m, b, kc, vc)[:, : m.heads * m.vdim]
    rows = [i for i in range(n) if T - n + i >= far]
    assert torch.allclose(got[rows], want[rows], atol=1e-3)
    hidden = [i for i in range(n) if T - n + i < far]
    assert not hidden or (got[hidden] - want[hidden]).abs().max() > 1e-2


def test_trace_runner(tmp_path, monkeypatch, capsys):
    from rl_b200.tools.trace_run import main

    cfg = R.CASES["all"]
    w = R.weights(cfg, 2)
    path = R.save(cfg, w, tmp_path / "m")
    a, b = R.tokens(cfg, 21, 1), R.tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:20], "want": [0, 19]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[20:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert main(["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    za, zb = R.oracle(cfg, w, a), R.oracle(cfg, w, b)

    def read(n):
        return torch.frombuffer(bytearray((tmp_path / "o" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    assert R.gap(read(0), torch.stack([za[0], za[19], zb[0]])) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    assert R.gap(read(2), torch.stack([zb[8], za[20]])) < TOL
