"""Kikivik (pre-norm layer-list models: latent attention with a query latent, chunked grouped attention with mixed values, clamped units,
experts weighted on their inputs) on the CPU: every mechanism and the whole engine against the float64 statement in ``kikivik_oracle``."""

import copy
import io
import json
import sys

import kikivik_cases as K
import kikivik_oracle as O
import pytest
import torch

from rl_b200.engine.engine import SamplingParams
from rl_b200.models.config import KIKIVIK_TRAITS, ModelConfig, preset, rotary_table
from rl_b200.models.gated import GatedExperts, GatedUnit
from rl_b200.models.hf_io import load_pretrained, save_pretrained
from rl_b200.models.mixers import GroupedAttentionMixer, LatentAttentionMixer, rotate_pairs
from rl_b200.models.transformer import PackedBatch, build_model
from rl_b200.ops import engine_ops as E
from rl_b200.ops import layer_ops as Y
from rl_b200.ops import sequence_ops as S

TOL = 3e-4        # (fp32 against float64; the small random models amplify roundings)
F64 = torch.float64


class Cfg:
    rms_norm_eps = 1e-4
    hidden_size = 56


def build(entry, dtype=torch.float32, device="cpu", cfg=Cfg):
    """The mixer of a layer entry, as the layer builds it."""
    cls = {"attention": GroupedAttentionMixer, "latent_attention": LatentAttentionMixer}[entry["type"]]
    m = cls({**KIKIVIK_TRAITS[entry["type"]], **entry["mixer"]}, cfg, dtype, device)
    if not hasattr(m, "in_proj"):
        m.add_projections(cfg.hidden_size, dtype, device)
    return m


def unit(spec, dtype=torch.float32, device="cpu", cfg=Cfg):
    spec = {**KIKIVIK_TRAITS.get(spec["kind"], {}), **spec}
    return (GatedExperts if spec["kind"] == "moe" else GatedUnit)(spec, cfg, dtype, device)


@pytest.fixture(scope="module", params=sorted(K.CASES))
def case(request, tmp_path_factory):
    cfg = K.CASES[request.param]
    w = K.weights(cfg, seed=7)
    return cfg, w, K.load(cfg, w, tmp_path_factory.mktemp(request.param))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("entry", [K.latent(), K.latent(heads=1, dim=3, rot_dim=2, vdim=5, kv_rank=9, q_rank=11), K.latent(heads=4, dim=32, rot_dim=32, vdim=8, scale=1.0)])
def test_latent_attention_alone(entry):
    w = {k: v.to(F64) for k, v in O.below(K.weights(K.config([(entry, None)]), 3), "l0.mix.").items()}
    m = K.module_weights(build(entry), w)
    h = torch.randn(70, 56, dtype=F64)
    y = m.sequence(h.float() @ m.in_proj.t(), torch.arange(70), torch.tensor([0, 70]))
    got = y.double() @ m.out_proj[:, : y.shape[1]].double().t()
    assert torch.allclose(got, O.latent_attention(w, h, entry["mixer"], 1e-4), atol=3e-5)


@pytest.mark.parametrize("entry", [K.attention(), K.attention(size=0, factor=0), K.attention(heads=3, kv_heads=3, dim=5, vdim=9, rot_dims=4, size=1), K.attention(heads=8, kv_heads=2, rot_dims=0, size=69),
                                   K.attention(rot_dims=24, size=70, v_mix=False), K.attention(size=35)])
@pytest.mark.parametrize("mixed", [False, True])
def test_grouped_attention_alone(entry, mixed):
    w = {k: v.to(F64) for k, v in O.below(K.weights(K.config([(entry, None)]), 3), "l0.mix.").items()}
    m = K.module_weights(build(entry), w)
    h = torch.randn(70, 56, dtype=F64)
    mixed = mixed and m.v_mix
    old = torch.randn(70, m.kv_heads, m.vdim, dtype=F64)
    y = m.sequence(h.float() @ m.in_proj.t(), torch.arange(70), torch.tensor([0, 70]), old.view(70, -1).float() if mixed else None)
    got = y.double() @ m.out_proj[:, : y.shape[1]].double().t()
    assert torch.allclose(got, O.attention(w, h, entry["mixer"], 1e-4, [old] if mixed else []), atol=3e-5)


def test_rotation():
    rot = {"dims": 6, "base": 100.0, "scaling": {"factor": 2.5}}
    f, gain = rotary_table(rot)
    assert gain == 1.0 and torch.allclose(f.double(), torch.tensor(O.frequencies(rot), dtype=F64), rtol=1e-6)
    x = torch.randn(9, 2, 8, dtype=F64)
    got = rotate_pairs(x.float(), torch.arange(40, 49), f, gain, False)
    assert torch.allclose(got.double(), O.rotate(x, rot, first=40), atol=1e-5)
    assert torch.equal(got[..., 6:], x[..., 6:].float()) and not torch.allclose(got[..., :6], x[..., :6].float(), atol=1e-2)


def test_units_and_their_limits():
    h = torch.randn(30, 56, dtype=F64)
    for spec in (K.dense(), K.dense(ff=9, limit=0.3)):
        w = {k: v.to(F64) for k, v in O.below(K.weights(K.config([(K.latent(), spec)]), 1), "l0.mlp.").items()}
        m = K.module_weights(unit(spec), w)
        assert (h @ w["gate"].T).max() > spec["limit"] and (h @ w["up"].T).abs().max() > spec["limit"]
        for got in (m(h.float()), Y.unit(h.float(), m)):
            assert torch.allclose(got.double(), O.clamped_unit(w, h, spec["limit"]), atol=2e-5)


@pytest.mark.parametrize("spec", [K.moe(), K.moe(experts=5, top=1), K.moe(experts=6, top=6, shared=0), K.moe(experts=9, top=2, ff=3, shared=5)])
def test_experts_alone(spec):
    w = {k: v.to(F64) for k, v in O.below(K.weights(K.config([(K.latent(), spec)]), 5), "l0.mlp.").items()}
    m = K.module_weights(unit(spec), w)
    h = torch.randn(60, 56, dtype=F64)
    want = O.experts(w, h, spec)
    assert m.correction is None and torch.allclose(m(h.float()).double(), want, atol=3e-5)
    x, nw = torch.randn(60, 56), torch.rand(56)
    x1 = x.clone()
    got = Y.feed_forward_(x1, h.float(), m, None, 1.0, 1e-3, nw)
    assert torch.allclose(x1.double(), x.double() + want, atol=3e-5) and torch.allclose(got.double(), O.rms(x.double() + want, 1e-3) * nw.double(), atol=3e-5)


def test_weights_on_the_inputs_are_not_weights_on_the_outputs():
    spec = K.moe(experts=4, top=1, shared=0)
    w = {k: v.to(F64) for k, v in O.below(K.weights(K.config([(K.latent(), spec)]), 5), "l0.mlp.").items()}
    h = torch.randn(40, 56)
    a, b = K.module_weights(unit(spec), w), K.module_weights(GatedExperts(dict(spec, corrected=False), Cfg, torch.float32, "cpu"), w)
    assert (a(h) - b(h)).abs().max() > 0.1


def test_start_and_joins():
    table, w, nw = torch.randn(9, 24), torch.randn(24), torch.randn(24)
    ids = torch.tensor([3, 0, 8])
    x, h = Y.embed(ids, table, 2.5, w, 1e-3)
    assert torch.allclose(x, table[ids] * 2.5) and torch.allclose(h.double(), O.rms(table[ids].double() * 2.5, 1e-3) * w.double(), atol=1e-5)
    y, z = torch.randn(3, 24), torch.randn(3, 24)
    x1 = x.clone()
    h = Y.add_normed_(x1, y, None, 1.0, 1e-3, nw, also=z)
    assert torch.allclose(x1, x + y + z, atol=1e-6) and torch.allclose(h.double(), O.rms((x + y + z).double(), 1e-3) * nw.double(), atol=1e-5)


@pytest.mark.parametrize("chunk", [0, 1, 5, 16, 21, 64])
def test_paged_decode_sees_its_chunk(chunk):
    """The framework's paged decode operator with chunks, the plain and the batched gather form."""
    G, H, D, bs = 2, 4, 8, 16
    lens = torch.tensor([1, 16, 17, 42, 43, 63, 64, 0], dtype=torch.int32)
    kc, vc, q = torch.randn(9, G, bs, D), torch.randn(9, G, bs, D), torch.randn(len(lens), H * D)
    bt = torch.stack([torch.randperm(9)[:4] for _ in lens]).int()
    got = E.paged_decode(q, kc, vc, bt, lens, H, G, D, scale=0.7, chunk=chunk)
    again = E._paged_decode_gather(q, kc, vc, bt, lens, H, G, D, 0.7, torch.empty_like(got), chunk=chunk)
    assert torch.allclose(got, again, atol=1e-5)
    for i, n in enumerate(lens.tolist()):
        for h in range(H if n else 0):
            k, v = (c[bt[i].long(), h // 2].reshape(-1, D)[:n].double() for c in (kc, vc))
            want = O.attend(torch.cat([torch.zeros(n - 1, D, dtype=F64), q[i : i + 1, h * D : (h + 1) * D].double()]), k, v, 0.7, O.visible(n, chunk or None))[-1]
            assert torch.allclose(got[i, h * D : (h + 1) * D].double(), want, atol=1e-5)


@pytest.mark.parametrize("size", [0, 16, 20, 32, 63, 64])
@pytest.mark.parametrize("far", [0, 1, 15, 16, 19, 20, 31, 32, 47, 62, 63])
@pytest.mark.parametrize("n", [1, 2, 20, 64])
def test_one_key_far_away(far, n, size):
    m = build(K.attention(heads=4, kv_heads=2, dim=16, vdim=8, rot_dims=0, factor=0, scale=2.0, size=size, v_mix=False))
    p, b, kc, vc, want = K.standout_case(m, 64, 16, far, n)
    with torch.no_grad():
        got = S.attention(p, m, b, kc, vc)[:, : m.heads * m.vdim].double()
    assert torch.allclose(got, want, atol=1e-3)


def test_the_oracle_tells_faults_apart():
    """Each planted fault of the statement moves some logits far beyond the tolerance of the tests here."""
    cfg = K.CASES["all"]
    w, toks = K.weights(cfg, 7), K.tokens(cfg, 70)
    want = K.oracle(cfg, w, toks)

    def changed(edit, weights=w):
        c = copy.deepcopy(cfg)
        edit(c)
        return K.gap(O.forward(c, weights, toks), want)

    def at(i, part, **kw):
        return lambda c: c["layers"][i][part].update(kw)

    faults = [at(0, "mixer", mask={"size": 25}), at(0, "mixer", mask={"size": 23}), at(3, "mixer", mask={"size": 18}), at(2, "mixer", mask=None),
              at(0, "mixer", rot={"dims": 16, "base": 1e4}), at(1, "mixer", rot={"dims": 6, "base": 5000.0}), at(1, "mixer", scale=0.26), at(1, "mlp", limit=1.3),
              at(0, "mlp", shared=None), at(4, "mlp", router={"experts": 7, "top": 2}), lambda c: c["norm"].update(eps=1e-2)]
    for i, f in enumerate(faults):
        assert changed(f) > 10 * TOL, i
    for leaf in ("l3.mix.vmix", "l1.mix.dq.norm", "l4.mix.dkv.norm", "l0.mix.k.norm"):
        assert changed(lambda c: None, {k: v * 1.05 if k == leaf else v for k, v in w.items()}) > 10 * TOL, leaf
    assert changed(lambda c: None, {k: v * 0 if k == "l0.mix.vmix" else v for k, v in w.items()}) == 0      # the first layer's share has no use


# ------------------------------------------------------------------------------------------------ model
def test_config_round_trip_and_checks(tmp_path):
    cfg = K.CASES["all"]
    c = ModelConfig.from_hf_dict(cfg)
    assert c.is_mixer and not c.is_recurrent and not c.caps_logits and c.layer_form == "pre"
    for name, k in K.CASES.items():
        c = ModelConfig.from_hf_dict(k)
        assert ModelConfig.from_hf_dict(json.loads(json.dumps(c.to_hf_dict()))) == c
        assert c.num_parameters() == sum(v.numel() for v in K.weights(k).values()), name
    w = K.weights(cfg, 1)
    m = K.load(cfg, w, tmp_path / "a")
    save_pretrained(m, str(tmp_path / "b"), dtype=torch.bfloat16)
    from safetensors.torch import load_file, save_file

    again = load_file(str(tmp_path / "b" / "model.safetensors"))
    assert set(again) == set(w) and all(torch.equal(again[k], w[k]) for k in w)
    l0, l1 = cfg["layers"][:2]
    for bad in (dict(l0, type="retention"), dict(l0, mixer={"heads": 2}), dict(l0, mixer=dict(l0["mixer"], kv_heads=3)), dict(l0, mixer=dict(l0["mixer"], mask={"size": 0})),
                dict(l0, mlp={"kind": "sparse", "ff": 3}), dict(l0, mlp=K.moe(experts=3, top=4)), dict(l1, mixer={k: v for k, v in l1["mixer"].items() if k != "q_rank"})):
        with pytest.raises(ValueError):
            ModelConfig.from_hf_dict(dict(cfg, layers=[bad]))
    with pytest.raises(ValueError):      # values of unequal size cannot be mixed
        ModelConfig.from_hf_dict(dict(cfg, layers=[l0, dict(l0, mixer=dict(l0["mixer"], vdim=8))]))
    with pytest.raises(KeyError):
        save_file({k: v for k, v in w.items() if k != "l1.mix.uq"}, str(tmp_path / "a" / "model.safetensors"))
        load_pretrained(str(tmp_path / "a"))


@pytest.mark.parametrize("ckpt", [False, True])
def test_trains(case, ckpt):
    cfg, w, model = case
    toks = K.tokens(cfg, 60)
    b = PackedBatch(torch.tensor(toks), torch.cat([torch.arange(22), torch.arange(38)]).int(), torch.tensor([0, 22, 60], dtype=torch.int32), 38)
    model.activation_checkpointing = ckpt
    z = model.logits(b)
    want = torch.cat([K.oracle(cfg, w, toks[:22]), K.oracle(cfg, w, toks[22:])])
    assert K.gap(z.detach(), want) < TOL
    lp = model.next_token_logprobs(b)
    lp = lp[0] if isinstance(lp, tuple) else lp
    ref = torch.log_softmax(want, -1)
    assert torch.allclose(lp[1:22].double(), ref[:21].gather(-1, torch.tensor(toks[1:22])[:, None])[:, 0], atol=1e-3)
    lp.sum().backward()
    mixing = [i for i, e in enumerate(cfg["layers"]) if e["mixer"].get("v_mix")]
    for n, p in model.named_parameters():
        if not (mixing and n == f"layers.{mixing[0]}.mixer.v_share"):      # (the first layer that mixes has nothing to mix with)
            assert p.grad is not None and torch.isfinite(p.grad).all(), n
    model.zero_grad(set_to_none=True)
    model.activation_checkpointing = False


def test_worker_trains_and_generates():
    from rl_b200.algorithms.loss.loss_functions import NLLLossFn
    from rl_b200.distributed.batched_data_dict import BatchedDataDict
    from rl_b200.policy.worker import PolicyWorker
    from rl_b200.utils.flops import model_flops

    mc = preset("tiny-kikivik")
    assert model_flops(mc, 20) > 0
    p = PolicyWorker(dict(precision="float32", train_global_batch_size=4, train_micro_batch_size=2, max_total_sequence_length=64,
                          optimizer=dict(name="torch.optim.AdamW", kwargs=dict(lr=1e-3)),
                          generation=dict(max_new_tokens=8, stop_token_ids=[], kv_cache_tokens=1024, block_size=16, max_running=4)),
                     model_cfg=mc, device="cpu", init_reference_model=False)
    recs = p.build_generation().engine.generate([K.tokens({"vocab": 264}, 12, s) for s in range(4)], SamplingParams(max_new_tokens=8, seed=1))
    ids = torch.tensor([r.prompt + r.out_tokens for r in recs])
    data = BatchedDataDict(input_ids=ids, input_lengths=torch.full((4,), 20), token_mask=torch.ones(4, 20), sample_mask=torch.ones(4))
    lp = p.get_logprobs(data)["logprobs"][:, 12:]
    assert torch.allclose(lp, torch.tensor([r.out_logprobs for r in recs]), atol=1e-4)
    losses = [float(p.train(data, NLLLossFn(), gbs=4, mbs=2)["loss"]) for _ in range(3)]
    assert losses[2] < losses[0]


def test_random_init():
    m = build_model(preset("tiny-kikivik"), seed=3, dtype=torch.float32)
    assert (m.layers[0].norm1 == 1).all() and (m.layers[1].mixer.q_norm == 1).all() and m.layers[1].mixer.q_up.std() > 0.01 and float(m.layers[0].mixer.v_share.detach()) == 0.5
    assert build_model(preset("tiny-kikivik"), seed=3, dtype=torch.float32).layers[1].ff.down.equal(m.layers[1].ff.down)
    with pytest.raises(NotImplementedError):
        build_model(preset("tiny-kikivik"), pp_size=2)


# ------------------------------------------------------------------------------------------------ engine
@pytest.mark.parametrize("cuts", [[1000], [1], [2], [3], [16], [17, 2, 33, 1], [50, 1]])
def test_portions_equal_the_oracle(case, cuts):
    cfg, w, model = case
    toks = K.tokens(cfg, 70)
    eng = K.engine(model)
    assert K.gap(K.run_cut(eng, "a", toks, cuts), K.oracle(cfg, w, toks)) < TOL
    assert eng.sched.num_free_blocks == 24


def test_mixed_batches_and_reused_pages(case):
    cfg, w, model = case
    seqs = {f"r{i}": K.tokens(cfg, n, seed=i) for i, n in enumerate([60, 1, 33, 17, 48, 2, 80, 16])}
    steps = K.mixed_schedule({r: len(t) for r, t in seqs.items()}, seed=5)
    eng = K.engine(model, pages=K.live_pages(steps, 16))
    got = K.run_schedule(eng, steps, seqs)
    for r, t in seqs.items():
        assert K.gap(got[r], K.oracle(cfg, w, t)) < TOL, r
    assert not eng._step_ids and eng.sched.num_free_blocks == eng.num_blocks


def greedy(cfg, w, prompt, n):
    o = list(prompt)
    for _ in range(n):
        o.append(int(K.oracle(cfg, w, o)[-1].argmax()))
    return o[len(prompt) :]


def test_greedy_generation(case):
    """Through the scheduler, with portions and, for equal prompts, shared pages."""
    cfg, w, model = case
    prompts = [K.tokens(cfg, n, seed=n) for n in (1, 5, 16, 17, 40, 5)]
    prompts[5] = list(prompts[1])
    prompts.append(prompts[4][:33])
    eng = K.engine(model, requests=3, max_prefill_tokens=24)
    recs = eng.generate(prompts, SamplingParams(greedy=True, max_new_tokens=9))
    for p, r in zip(prompts, recs):
        assert r.out_tokens == greedy(cfg, w, p, 9)
    again = eng.generate(prompts[::-1], SamplingParams(greedy=True, max_new_tokens=9))
    assert [r.out_tokens for r in again[::-1]] == [r.out_tokens for r in recs]


def test_long_decoding_passes_chunks(case):
    """Decoding over several borders: the log-probabilities are those of the whole sequence at once."""
    cfg, w, model = case
    eng = K.engine(model, requests=2)
    recs = eng.generate([K.tokens(cfg, 3, 1), K.tokens(cfg, 20, 2)], SamplingParams(temperature=1.0, max_new_tokens=90, seed=3))
    for r in recs:
        z = K.oracle(cfg, w, r.prompt + r.out_tokens)[len(r.prompt) - 1 : -1]
        lp = torch.log_softmax(z, -1).gather(-1, torch.tensor(r.out_tokens)[:, None])[:, 0]
        assert torch.allclose(lp, torch.tensor(r.out_logprobs, dtype=F64), atol=2e-3)


def test_trace_runner(tmp_path, monkeypatch, capsys):
    from rl_b200.tools.trace_run import main

    cfg = K.CASES["all"]
    w = K.weights(cfg, 2)
    path = K.save(cfg, w, tmp_path / "m")
    a, b = K.tokens(cfg, 31, 1), K.tokens(cfg, 9, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}, {"id": "b", "tokens": b[:1], "want": [0]}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[1:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[8:], "want": [0]}, {"id": "a", "tokens": a[30:], "want": [0]}], "end": ["a", "b"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in steps) + "\n"))
    assert main(["--model", path, "--dtype", "float32", "--out", str(tmp_path / "o"), "--max-tokens", "128", "--device", "cpu"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    za, zb = K.oracle(cfg, w, a), K.oracle(cfg, w, b)

    def read(n):
        return torch.frombuffer(bytearray((tmp_path / "o" / f"{n}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])

    assert K.gap(read(0), torch.stack([za[0], za[29], zb[0]])) < TOL
    assert not (tmp_path / "o" / "1.f32").exists()
    assert K.gap(read(2), torch.stack([zb[8], za[30]])) < TOL
