"""Zonidra (layer-list models with norms on both sides of the sublayers, token shift, windowed sigmoid attention on shared keys, polynomial units,
experts with identity outputs, pair embeddings) on the CPU: every mechanism and the whole engine against the float64 statement in
``zonidra_oracle``."""

import copy
import io
import json
import sys

import pytest
import torch
import zonidra_cases as Z
import zonidra_oracle as O

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import ZONIDRA_TRAITS, ModelConfig, preset, rotary_table
from rl_b200.models.gated import feed_forward, poly_norm
from rl_b200.models.hf_io import load_pretrained, save_pretrained
from rl_b200.models.mixers import GroupedAttentionMixer, rotate_pairs
from rl_b200.models.transformer import PackedBatch, build_model
from rl_b200.ops import layer_ops as Y
from rl_b200.ops import mixer_ops as X
from rl_b200.ops import sequence_ops as S

TOL = 3e-4        # (fp32 against float64; the small random models amplify roundings)
F64 = torch.float64


class Cfg:
    rms_norm_eps = 1e-4
    hidden_size = 56


def build(entry, dtype=torch.float32, device="cpu", cfg=Cfg):
    """The mixer of a layer entry, as the layer builds it."""
    return GroupedAttentionMixer({**ZONIDRA_TRAITS["attention"], **entry["mixer"]}, cfg, dtype, device)


def unit(spec, dtype=torch.float32, device="cpu", cfg=Cfg):
    return feed_forward({**ZONIDRA_TRAITS[spec["kind"]], **spec}, cfg, dtype, device)


def part(layers, prefix, seed=3, **kw):
    """Tensors below ``prefix`` of a random model of these layers, in float64."""
    return {k: v.to(F64) for k, v in O.below(Z.weights(Z.config(layers, **kw), seed), prefix).items()}


@pytest.fixture(scope="module", params=sorted(Z.CASES))
def case(request, tmp_path_factory):
    cfg = Z.CASES[request.param]
    w = Z.weights(cfg, seed=7)
    return cfg, w, Z.load(cfg, w, tmp_path_factory.mktemp(request.param))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("scaling", [None, Z.LONG, dict(factor=8.0, low=0.5, high=2.0, original=30), dict(factor=2.0, low=1.0, high=4.0, original=100000)])
def test_rotation(scaling):
    rot = {"dims": 12, "base": 100.0, "scaling": scaling}
    f, gain = rotary_table(rot)
    assert gain == 1.0 and torch.allclose(f.double(), torch.tensor(O.frequencies(rot), dtype=F64), rtol=1e-6)
    x = torch.randn(9, 2, 14, dtype=F64)
    got = rotate_pairs(x.float(), torch.arange(40, 49), f, gain, False)
    assert torch.allclose(got.double(), O.rotate(x, rot, first=40), atol=1e-5)
    assert torch.equal(got[..., 12:], x[..., 12:].float())


def test_scaled_frequencies_fall_into_three_ranges():
    f = torch.tensor(O.frequencies({"dims": 16, "base": 1e4, "scaling": Z.LONG}), dtype=F64) / torch.tensor(O.frequencies({"dims": 16, "base": 1e4}), dtype=F64)
    assert (f == 1).any() and torch.isclose(f, torch.tensor(1 / 3.0, dtype=F64)).any() and ((f > 0.34) & (f < 0.99)).any()


@pytest.mark.parametrize("entry", [Z.attention(), Z.attention(size=0), Z.attention(heads=3, kv_heads=3, dim=5, vdim=9, rot_dims=4, size=1, keep=0), Z.attention(heads=8, kv_heads=2, rot_dims=0, size=69),
                                   Z.attention(rot_dims=24, size=10, keep=50), Z.attention(size=35, keep=0, scaling=None)])
@pytest.mark.parametrize("borrowed", [False, True])
def test_attention_alone(entry, borrowed):
    w = part([(entry, None)], "l0.mix.")
    m = Z.module_weights(build(entry), w)
    h, other = torch.randn(70, 56, dtype=F64), torch.randn(70, 56, dtype=F64)
    kv = None
    if borrowed:
        kv = O.keys_values(w, other, entry["mixer"])
        reader = build({"mixer": dict(entry["mixer"], kv_from=0)})
        assert not {"k", "v"} & {leaf for leaf, _ in reader.tensors()} and reader.in_width < m.in_width
        m = Z.module_weights(reader, w)
    y = m.sequence(h.float() @ m.in_proj.t(), torch.arange(70), torch.tensor([0, 70]), None, None if kv is None else tuple(t.float() for t in kv))
    got = y.double() @ m.out_proj[:, : y.shape[1]].double().t()
    assert torch.allclose(got, O.attention(w, h, entry["mixer"], kv)[0], atol=5e-5)


def test_poly_units():
    h = torch.randn(30, 56, dtype=F64)
    for spec in (Z.dense(), Z.dense(ff=9), Z.dense(ff=1)):
        w = part([(Z.attention(), spec)], "l0.mlp.", 1)
        m = Z.module_weights(unit(spec), w)
        for got in (m(h.float()), Y.poly_unit(h.float(), m)):
            assert torch.allclose(got.double(), O.poly_unit(w, h, 1e-4), atol=2e-5)
    z, c = torch.randn(5, 12, dtype=F64), torch.randn(4, dtype=F64)
    assert torch.allclose(poly_norm(z.float(), c.float(), 1e-3).double(), O.poly_norm(z, c, 1e-3), atol=1e-5)
    x = torch.cat([z, torch.full((5, 4), 7.0, dtype=F64)], 1).float()
    Y.poly_norm_(x, c.float(), 12, 1e-3)
    assert torch.allclose(x[:, :12].double(), O.poly_norm(z, c, 1e-3), atol=1e-5) and (x[:, 12:] == 7).all()


@pytest.mark.parametrize("spec", [Z.moe(), Z.moe(experts=5, identity=0, top=1), Z.moe(experts=6, identity=1, top=7, shared=0), Z.moe(experts=2, identity=9, top=2, ff=3, shared=5, scale=1.0), Z.moe(scale=0.3)])
def test_experts_alone(spec):
    w = part([(Z.attention(), spec)], "l0.mlp.", 5)
    m = Z.module_weights(unit(spec), w)
    h = torch.randn(60, 56, dtype=F64)
    want = O.experts(w, h, spec)
    assert torch.allclose(m(h.float()).double(), want, atol=5e-5)
    x, nw, ow, ls = torch.randn(60, 56), torch.rand(56), torch.rand(56), torch.rand(56)
    x1, got = Y.feed_forward(x.clone(), h.float(), m, ow, 1.0, 1e-3, nw, ls)
    new = x.double() + O.rms(want, 1e-3) * ow.double() * ls.double()
    assert torch.allclose(x1.double(), new, atol=3e-5) and torch.allclose(got.double(), O.rms(new, 1e-3) * nw.double(), atol=3e-5)


def test_corrections_choose_and_do_not_weigh():
    spec = Z.moe(experts=4, identity=2, top=2, shared=0)
    w = part([(Z.attention(), spec)], "l0.mlp.", 5)
    h = torch.randn(40, 56, dtype=F64)
    m = Z.module_weights(unit(spec), w)
    z = h.float() @ w["router"].float().T
    wt, idx = m.choose(z)
    assert torch.allclose(wt, torch.softmax(z, -1).gather(1, idx) * 1.7, atol=1e-6)
    chosen = [{e for e, _ in c} for c in O.route(w, h, spec["router"])]
    assert all(set(i.tolist()) == c for i, c in zip(idx, chosen))
    plain = [{e for e, _ in c} for c in O.route(dict(w, correction=w["correction"] * 0), h, spec["router"])]
    assert chosen != plain and any(max(c) >= 4 for c in chosen)


def pieces(lens, starts, states, tokens, device="cpu", dtype=torch.int64):
    """Batch of pieces (single tokens first), with what the operators that look at the token before need."""
    n_single = sum(n == 1 for n in lens)
    pos = torch.cat([torch.arange(s, s + n) for n, s in zip(lens, starts)]).int()
    off = torch.cat([torch.arange(n) for n in lens]).int()
    st = torch.tensor(states)
    cu = torch.tensor([0] + list(lens[n_single:])).cumsum(0).int() if n_single < len(lens) else None
    b = X.TokenBatch(ids=torch.tensor(tokens, dtype=dtype, device=device), positions=pos.to(device), slots=None, n_single=n_single, n_paged=0, block_table=None, seq_lens=None,
                     state_rows=st.to(device), cu=cu.to(device) if cu is not None else None)
    if cu is not None:
        b.row_off, b.row_state = off.to(device), st.repeat_interleave(torch.tensor(lens)).to(device)
    return b


def shift_schedule(seed=0):
    """Steps over three sequences: (lens, starts, state rows) with single tokens first; a sequence leaves a step out, a state row is used again."""
    return [([1, 4], [0, 0], [2, 1]), ([1, 2, 5], [1, 4, 0], [2, 1, 3]), ([1, 1], [6, 5], [1, 3]), ([1, 3, 2], [2, 0, 6], [2, 1, 3])]


@pytest.mark.parametrize("bigram", [(13, 5, 3), None])
@pytest.mark.parametrize("d", [8, 7])
def test_start_and_shift_over_steps(bigram, d, device="cpu", dt=torch.float32, tol=1e-5):
    """The start of the stream and a join, cut into steps, beside whole sequences. (The GPU tests run the same on the kernels.)"""
    g = torch.Generator().manual_seed(0)
    rnd = lambda *s: torch.randn(*s, generator=g).to(dt).to(device)   # noqa: E731
    table, pairs, norm, s0, s1, w, ls, nw = rnd(20, d), rnd(14, d), rnd(d), rnd(d), rnd(d), rnd(d), rnd(d), rnd(d)
    big = dict(zip(("buckets", "mul_prev", "mul_cur"), bigram)) if bigram else None
    carry = Y.Carry(4, 2, d, bool(bigram), device)
    if carry.state is not None:
        carry.state.fill_(9.0)
    seqs, runs, got = {}, [], {}
    for lens, starts, states in shift_schedule():
        toks, ys = [], []
        for n, s, st in zip(lens, starts, states):
            if s == 0:
                seqs[st] = len(runs)
                runs.append(([], []))
            t, y = torch.randint(0, 20, (n,), generator=g).tolist(), torch.randn(n, d, generator=g).to(dt)
            runs[seqs[st]][0].extend(t)
            runs[seqs[st]][1].append(y)
            toks += t
            ys.append(y)
        b = pieces(lens, starts, states, toks, device, torch.int32 if device != "cpu" else torch.int64)
        x, h = Y.start(b, table, 1.5, norm, 1e-3, pairs if bigram else None, big, Y.Shift(s0, 0, carry, b))
        x1, h1 = Y.join(x.clone(), torch.cat(ys).to(device), w, 1.0, 1e-3, nw, ls=ls, shift=Y.Shift(s1, 1, carry, b))
        carry.commit(b)
        at = 0
        for n, st in zip(lens, states):
            got.setdefault(seqs[st], []).append([t[at : at + n].double().cpu() for t in (x, h, x1, h1)])
            at += n
    c = lambda t: t.double().cpu()   # noqa: E731
    for i, (t, ys) in enumerate(runs):
        x = c(table)[torch.tensor(t)] * 1.5
        if bigram:
            x = x + c(pairs)[torch.tensor(O.pair_rows(t, big))]
        h = O.shift(O.rms(x, 1e-3) * c(norm), c(s0))
        x1 = x + O.rms(c(torch.cat(ys)), 1e-3) * c(w) * c(ls)
        h1 = O.shift(O.rms(x1, 1e-3) * c(nw), c(s1))
        for q, want in enumerate((x, h, x1, h1)):
            res = torch.cat([p[q] for p in got[i]])
            assert torch.allclose(res, want, atol=(1e-5 if q in (0, 2) else tol) * 10, rtol=tol), (i, q)


@pytest.mark.parametrize("source", [None, 0])
@pytest.mark.parametrize("size,keep", [(0, 0), (16, 0), (20, 5), (1, 1), (1, 16), (63, 1), (64, 0), (10, 50)])
@pytest.mark.parametrize("n", [1, 2, 20, 64])
def test_one_key_far_away(size, keep, n, source):
    for far in {0, 1, keep - 1, keep, 15, 16, 31, 32, 47, 62, 63, 63 - size, 64 - size} & set(range(64)):
        m = build(Z.attention(heads=4, kv_heads=2, dim=16, vdim=8, rot_dims=0, scale=2.0, size=size, keep=keep, source=source))
        p, b, kc, vc, want = Z.standout_case(m, 64, 16, far, n)
        with torch.no_grad():
            got = S.attention(p, m, b, kc, vc)[:, : m.heads * m.vdim].double()
        assert torch.allclose(got, want, atol=1e-4) and (want.abs().amax(-1) > 0.1).any() == bool(O.visible(64, {"size": size or 64, "keep_first": keep})[64 - n :, far].any())


def test_the_oracle_tells_faults_apart():
    """Each planted fault of the statement moves some logits far beyond the tolerance of the tests here."""
    cfg = Z.CASES["all"]
    w, toks = Z.weights(cfg, 7), Z.tokens(cfg, 70)
    want = Z.oracle(cfg, w, toks)

    def changed(edit, weights=w):
        c = copy.deepcopy(cfg)
        edit(c)
        return Z.gap(O.forward(c, weights, toks), want)

    def at(i, key, **kw):
        return lambda c: c["layers"][i][key].update(kw)

    rot = {"dims": 16, "base": 1e4}
    faults = [at(0, "mixer", mask={"size": 25, "keep_first": 3}), at(0, "mixer", mask={"size": 23, "keep_first": 3}), at(0, "mixer", mask={"size": 24, "keep_first": 2}), at(0, "mixer", mask={"size": 24, "keep_first": 4}),
              at(3, "mixer", mask={"size": 17, "keep_first": 20}), at(2, "mixer", mask=None), at(0, "mixer", rot=rot), at(0, "mixer", rot=dict(rot, scaling=dict(Z.LONG, high=3.0))),
              at(0, "mixer", rot=dict(rot, scaling=dict(Z.LONG, low=2.0))), at(3, "mixer", kv_from=1), at(1, "mixer", scale=0.31), at(0, "mlp", shared=None), at(4, "mlp", router={"experts": 7, "top": 2, "scale": 1.7}),
              at(0, "mlp", router={"experts": 7, "identity": 2, "top": 3, "scale": 1.75}), lambda c: c["norm"].update(eps=1e-2), lambda c: c["embedding"].update(scale=2.0),
              lambda c: c["embedding"]["bigram"].update(mul_cur=6), lambda c: c["embedding"]["bigram"].update(buckets=100)]
    for i, f in enumerate(faults):
        if i == 9:      # (layer 1 has no keys of its own: it hands on those of layer 0)
            assert changed(f) == 0
            continue
        assert changed(f) > 10 * TOL, i
    for leaf in ("l0.shift", "l3.shift", "l1.ls1", "l1.ls2", "l2.norm1b", "l4.norm2b", "l2.mix.pb", "l0.mlp.correction", "l1.mlp.act", "l0.mlp.shared.sg", "l3.mix.g", "bigram"):
        assert changed(lambda c: None, {k: v * 1.2 if k == leaf else v for k, v in w.items()}) > 10 * TOL, leaf


# ------------------------------------------------------------------------------------------------ model
def test_config_round_trip_and_checks(tmp_path):
    cfg = Z.CASES["all"]
    c = ModelConfig.from_hf_dict(cfg)
    assert c.is_mixer and c.is_recurrent and not c.caps_logits and c.layer_form == "pre"
    for name, k in Z.CASES.items():
        c = ModelConfig.from_hf_dict(k)
        assert ModelConfig.from_hf_dict(json.loads(json.dumps(c.to_hf_dict()))) == c
        assert c.num_parameters() == sum(v.numel() for v in Z.weights(k).values()), name
    w = Z.weights(cfg, 1)
    m = Z.load(cfg, w, tmp_path / "a")
    save_pretrained(m, str(tmp_path / "b"), dtype=torch.bfloat16)
    from safetensors.torch import load_file, save_file

    again = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(again) == set(w) and all(torch.equal(again[k], w[k]) for k in w)
    l0, l1 = cfg["layers"][:2]
    for bad in (dict(l0, type="retention"), dict(l0, mixer={"heads": 2}), dict(l0, mixer=dict(l0["mixer"], kv_heads=3)), dict(l0, mixer=dict(l0["mixer"], mask={"size": 0})),
                dict(l0, mlp={"kind": "sparse", "ff": 3}), dict(l0, mlp=Z.moe(experts=3, identity=1, top=5)), l1):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[bad]))
    for kw in (dict(vdim=8), dict(kv_from=1), dict(kv_from=2)):      # unequal sizes, a layer without keys of its own, a layer behind
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[l0, l1, dict(l1, mixer=dict(l1["mixer"], **kw))]))
    with pytest.raises(KeyError):
        save_file({k: v for k, v in w.items() if k != "l1.ls2"}, str(tmp_path / "a" / "model.safetensors"))
        load_pretrained(str(tmp_path / "a"))


@pytest.mark.parametrize("ckpt", [False, True])
def test_trains(case, ckpt):
    cfg, w, model = case
    toks = Z.tokens(cfg, 60)
    b = PackedBatch(torch.tensor(toks), torch.cat([torch.arange(22), torch.arange(38)]).int(), torch.tensor([0, 22, 60], dtype=torch.int32), 38)
    model.activation_checkpointing = ckpt
    z = model.logits(b)
    want = torch.cat([Z.oracle(cfg, w, toks[:22]), Z.oracle(cfg, w, toks[22:])])
    assert Z.gap(z.detach(), want) < TOL
    lp = model.next_token_logprobs(b)
    lp = lp[0] if isinstance(lp, tuple) else lp
    ref = torch.log_softmax(want, -1)
    assert torch.allclose(lp[1:22].double(), ref[:21].gather(-1, torch.tensor(toks[1:22])[:, None])[:, 0], atol=1e-3)
    lp.sum().backward()
    for n, p in model.named_parameters():
        assert p.grad is not None and torch.isfinite(p.grad).all(), n
    model.zero_grad(set_to_none=True)
    model.activation_checkpointing = False


def test_worker_trains_and_generates():
    from rl_b200.algorithms.loss.loss_functions import NLLLossFn
    from rl_b200.distributed.batched_data_dict import BatchedDataDict
    from rl_b200.policy.worker import PolicyWorker
    from rl_b200.utils.flops import model_flops

    mc = preset("tiny-zonidra")
    assert 0 < model_flops(mc, 10) < model_flops(mc, 40)
    p = PolicyWorker(dict(precision="float32", train_global_batch_size=4, train_micro_batch_size=2, max_total_sequence_length=64,
                          optimizer=dict(name="torch.optim.AdamW", kwargs=dict(lr=1e-3)),
                          generation=dict(max_new_tokens=8, stop_token_ids=[], kv_cache_tokens=1024, block_size=16, max_running=4)),
                     model_cfg=mc, device="cpu", init_reference_model=False)
    recs = p.build_generation().engine.generate([Z.tokens({"vocab": 264}, 12, s) for s in range(4)], SamplingParams(max_new_tokens=8, seed=1))
    ids = torch.tensor([r.prompt + r.out_tokens for r in recs])
    data = BatchedDataDict(input_ids=ids, input_lengths=torch.full((4,), 20), token_mask=torch.ones(4, 20), sample_mask=torch.ones(4))
    lp = p.get_logprobs(data)["logprobs"][:, 12:]
    assert torch.allclose(lp, torch.tensor([r.out_logprobs for r in recs]), atol=1e-4)
    losses = [float(p.train(data, NLLLossFn(), gbs=4, mbs=2)["loss"]) for _ in range(3)]
    assert losses[2] < losses[0]


def test_random_init():
    m = build_model(preset("tiny-zonidra"), seed=3, dtype=torch.float32)
    l0, l1 = m.layers[0], m.layers[1]
    assert (l0.norm1b == 1).all() and (l0.ls1 == 1).all() and l0.mixer.q_norm is None and l0.lends and not l1.lends and m.bigram.std() > 0.01
    assert l1.mixer.kv_from == 0 and torch.allclose(l0.mixer.offset, -torch.log(torch.tensor(20.0))) and l1.ff.coef.sum() == 1
    assert build_model(preset("tiny-zonidra"), seed=3, dtype=torch.float32).layers[1].ff.down.equal(m.layers[1].ff.down)
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-zonidra"), pp_size=2)


# ------------------------------------------------------------------------------------------------ engine
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3], [16], [17, 2, 33, 1], [50, 1]])
def test_portions_equal_the_oracle(case, cuts):
    cfg, w, model = case
    toks = Z.tokens(cfg, 70)
    eng = Z.engine(model)
    assert Z.gap(Z.run_cut(eng, "a", toks, cuts), Z.oracle(cfg, w, toks)) < TOL
    assert eng.sched.num_free_blocks == 24


def test_mixed_batches_and_reused_pages(case):
    """More requests than state rows and pages: both are used again."""
    cfg, w, model = case
    seqs = {f"r{i}": Z.tokens(cfg, n, seed=i) for i, n in enumerate([60, 1, 33, 17, 48, 2, 80, 16])}
    steps = Z.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = Z.engine(model, pages=Z.live_pages(steps, 16))
    got = Z.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert Z.gap(got[r], Z.oracle(cfg, w, t)) < TOL, r
    assert not eng._step_ids and eng.sched.num_free_blocks == eng.num_blocks and len(eng._free_rows) == 4


def test_borrowing_layers_have_no_pages(case):
    cfg, _, model = case
    eng = Z.engine(model)
    eng.wake()
    for i, e in enumerate(cfg["layers"]):
        src = e["mixer"].get("kv_from")
        assert src is None or (eng.k_cache[i] is eng.k_cache[src] and eng._cache_width(i) == 0)
    own = sum(e["mixer"]["kv_heads"] * (e["mixer"]["dim"] + e["mixer"]["vdim"]) for e in cfg["layers"] if e["mixer"].get("kv_from") is None)
    assert eng.kv_cache_bytes() == own * 24 * 16 * 4


def greedy(cfg, w, prompt, n):
    o = list(prompt)
    for _ in range(n):
        o.append(int(Z.oracle(cfg, w, o)[-1].argmax()))
    return o[len(prompt) :]


def test_greedy_generation(case):
    """Through the scheduler, with portions and equal prompts."""
    cfg, w, model = case
    prompts = [Z.tokens(cfg, n, seed=n) for n in (1, 5, 16, 17, 40, 5)]
    prompts[5] = list(prompts[1])
    prompts.append(prompts[4][:33])
    eng = Z.engine(model, requests=3, max_prefill_tokens=24)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=9))
    for p, r in zip(prompts, recs):
        assert r.out_tokens == greedy(cfg, w, p, 9)
    again = eng.generate(prompts[::-1], SamplingParams(greedy=True, max_new_tokens=9))
    assert [r.out_tokens for r in again[::-1]] == [r.out_tokens for r in recs]


def test_long_decoding_passes_windows(case):
    """Decoding until the window has left the prompt: the log-probabilities are those of the whole sequence at once."""
    cfg, w, model = case
    eng = Z.engine(model, requests=2)
    recs = eng.generate([Z.tokens(cfg, 3, 1), Z.tokens(cfg, 20, 2)], SamplingParams(temperature=1.0, max_new_tokens=90, seed=3))
    for r in recs:
        z = Z.oracle(cfg, w, r.prompt + r.out_tokens)[len(r.prompt) - 1 : -1]
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert torch.allclose(lp, torch.tensor(r.out_logprobs, dtype=F64), atol=2e-3)


def test_trace_runner(tmp_path, monkeypatch, capsys):
    from rl_b200.tools.trace_run import main

    cfg = Z.CASES["all"]
    w = Z.weights(cfg, 2)
    path = Z.save(cfg, w, tmp_path / "m")
    a, b = Z.tokens(cfg, 31, 1), Z.tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[30:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert main(["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    za, zb = Z.oracle(cfg, w, a), Z.oracle(cfg, w, b)

    def read(n):
        return torch.frombuffer(bytearray((tmp_path / "o" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    assert Z.gap(read(0), torch.stack([za[0], za[29], zb[0]])) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    assert Z.gap(read(2), torch.stack([zb[8], za[30]])) < TOL
