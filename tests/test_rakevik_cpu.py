"""Rakevik against a plain restatement of its equations, on the CPU path: mechanisms, caches, batches, generation."""

import oracle_rakevik as O
import pytest
import rakevik_cases as C
import torch

from easydel_b200.ops import ssm, stream

TOL = 2e-5


def _r(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
def test_token_shift_and_norm_carry_a_row_between_steps():
    x, w, mu = _r(9, 12), 1 + 0.1 * _r(12, seed=1), torch.rand(12)
    want = O.token_shift(O.rms_norm(x, w, 1e-5), mu)
    cu = torch.tensor([0, 9], dtype=torch.int32)
    assert torch.allclose(stream.norm_shift(x, w, 1e-5, torch.float32, mu, cu), want, atol=1e-6)
    state, slots = torch.zeros(3, 12), torch.tensor([2], dtype=torch.int32)
    parts, at = [], 0
    for n in (2, 1, 4, 2):
        parts.append(stream.norm_shift(x[at:at + n], w, 1e-5, torch.float32, mu,
                                       torch.tensor([0, n], dtype=torch.int32), slots, state))
        at += n
    assert torch.allclose(torch.cat(parts), want, atol=1e-6)
    assert torch.allclose(state[2], O.rms_norm(x, w, 1e-5)[-1], atol=1e-6) and not state[:2].any()


def test_xielu_both_branches():
    z = torch.cat([_r(50) * 3, torch.tensor([0.0, -1e-4, 1e-4, -30.0])])
    for act in (torch.tensor([0.3, -1.2]), torch.tensor([-2.0, 1.5])):
        assert torch.allclose(stream.xielu(z, act), O.xielu(z, act), rtol=1e-5, atol=1e-6)


def test_hgrn2_scan_and_forget_gate():
    H, D, V, T = 2, 5, 7, 11
    proj, b, low = _r(T, 2 * H * D + H * V), _r(H * D, seed=1), torch.rand(H * D)
    q, z, v = torch.split(proj, [H * D, H * D, H * V], -1)
    f = O.forget_gate(z, b, low).view(T, H, D)
    want, end = O.hgrn2_scan((q * O.sigmoid(q)).view(T, H, D), f, v.reshape(T, H, V))
    norm = 1 + 0.1 * _r(V, seed=2)
    state = torch.zeros(1, H, D, V)
    got = ssm.hgrn2(proj, (H, D, V), b, low, norm, 1e-6, torch.tensor([0, T], dtype=torch.int32), T, None, state)
    assert torch.allclose(got.view(T, H, V), O.rms_norm(want, norm, 1e-6), atol=1e-5)
    assert torch.allclose(state[0], end, atol=1e-6)


def test_query_temperature_steps_at_multiples():
    p = torch.arange(40)
    got = stream.query_temperature(p, (0.4, 10))
    assert torch.allclose(got, O.query_temperature(p.float(), 0.4, 10))
    assert got[8] == got[0] and got[9] > got[8] and got[18] == got[9] and got[19] > got[18]


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_logits_and_hidden_states(tmp_path, name):
    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    toks = C.tokens(37, cfg["vocab"])
    res = []
    want = O.forward(cfg, w, toks, residuals=res)
    with torch.no_grad():
        out = model(input_ids=torch.tensor([toks]), output_hidden_states=True)
    assert C.error(out.logits[0], want) < TOL
    runs = model.model.layer_runs
    assert len(out.hidden_states) == len(res) + 1 == (len(runs) if runs else len(cfg["layers"])) + 1
    last = O.rms_norm(res[-1], w["final.norm"].double(), cfg["norm"]["eps"])
    assert torch.allclose(out.hidden_states[-1][0].double(), last, atol=1e-3)
    with torch.enable_grad():      # the differentiable form: no cache, batch of two equal rows
        lg = model(input_ids=torch.tensor([toks, toks[::-1]])).logits
        assert C.error(lg[0], want) < TOL
        assert C.error(lg[1], O.forward(cfg, w, toks[::-1])) < TOL
        lg.square().mean().backward()
    assert all(p.grad is not None for p in model.parameters())


@pytest.mark.parametrize("mutate", ["no_shift", "no_sink", "no_q_temp", "kv_head", "no_loop_step"])
def test_a_wrong_mechanism_would_show(tmp_path, mutate):
    """The comparison is sharp enough to notice each of these mistakes (planted in the oracle)."""
    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cpu")
    toks = C.tokens(30, cfg["vocab"])
    with torch.no_grad():
        got = model(input_ids=torch.tensor([toks])).logits[0]
    assert C.error(got, O.forward(cfg, w, toks)) < TOL
    assert C.error(got, O.forward(cfg, w, toks, mutate=mutate)) > 100 * TOL


@pytest.mark.parametrize("name", ["looped", "odd", "recurrent"])
@pytest.mark.parametrize("cuts", [[140, 1], [2], [127, 2, 1, 3], [1]])
def test_portions_and_decoding_match_the_whole(tmp_path, name, cuts):
    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    toks = C.tokens(145 if cuts != [1] else 20, cfg["vocab"], 3)
    want = O.forward(cfg, w, toks)
    assert C.error(C.run_cut(C.replayer(model), "a", toks, cuts), want) < TOL


def test_mixed_batches_reuse_pages_and_slots(tmp_path):
    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cpu")
    rep = C.replayer(model, max_tokens=512, max_requests=3)
    pool_free = [m.pool.num_free for m in rep.engine.kv.managers]
    seqs = {n: C.tokens(k, cfg["vocab"], i) for i, (n, k) in enumerate(
        [("a", 131), ("b", 5), ("c", 90), ("d", 129), ("e", 2)])}
    got, at = {n: [] for n in seqs}, {n: 0 for n in seqs}
    plan = [[("a", 60), ("b", 1)], [("a", 70), ("b", 2), ("c", 64)], [("b", 2), ("a", 1)], [("c", 1), ("d", 100)],
            [("d", 2), ("c", 25), ("e", 1)], [("d", 27), ("e", 1)]]
    for step in plan:
        entries, end = [], []
        for n, k in step:
            entries.append({"id": n, "tokens": seqs[n][at[n]:at[n] + k], "want": list(range(k))})
            at[n] += k
            if at[n] == len(seqs[n]):
                end.append(n)
        lg = rep.step(entries, end)
        for n, k in step:
            got[n].append(lg[:k])
            lg = lg[k:]
    for n, toks in seqs.items():
        assert at[n] == len(toks)
        assert C.error(torch.cat(got[n]), O.forward(cfg, w, toks)) < TOL, n
    assert [m.pool.num_free for m in rep.engine.kv.managers] == pool_free
    assert len(rep.engine._free_slots) == 3 and not rep.engine.scheduler.running


def test_replay_refuses_what_does_not_fit(tmp_path):
    cfg, w, model = C.make(tmp_path, "recurrent", torch.float32, "cpu")
    rep = C.replayer(model, max_tokens=128, max_requests=1)
    rep.step([{"id": "a", "tokens": [1, 2], "want": []}])
    with pytest.raises(RuntimeError, match="slots"):
        rep.step([{"id": "b", "tokens": [1], "want": []}])


# ------------------------------------------------------------------------------------------------ engine and checkpoints
def _greedy(cfg, w, prompt, n):
    toks = list(prompt)
    for _ in range(n):
        toks.append(int(O.forward(cfg, w, toks)[-1].argmax()))
    return toks[len(prompt):]


@pytest.mark.parametrize("async_scheduling", [False, True])
def test_greedy_generation_through_the_engine(tmp_path, async_scheduling):
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cpu")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (1, 13, 130, 40)]
    # few slots, a small token budget (prompts are cut) and few pages (a request is preempted and starts over)
    eng = eSurge(model, max_model_len=256, max_num_seqs=3, num_pages=4, max_num_batched_tokens=48,
                 async_scheduling=async_scheduling)
    assert eng.kv.num_groups == 2 and not eng.pool.enable_caching
    outs = eng.generate(prompts, SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == _greedy(cfg, w, p, 6)
    outs = eng.generate([prompts[1]], SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True))
    assert outs[0].outputs[0].token_ids == _greedy(cfg, w, prompts[1], 6)      # a slot that was used before
    sampled = eng.generate([prompts[1]], SamplingParams(max_tokens=5, temperature=0.8, top_k=5, seed=1))
    assert len(sampled[0].outputs[0].token_ids) <= 5


def test_generate_with_padding_and_beams(tmp_path):
    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cpu")
    a, b = C.tokens(9, cfg["vocab"], 1), C.tokens(5, cfg["vocab"], 2)
    ids = torch.tensor([a, [0] * 4 + b])
    mask = torch.tensor([[1] * 9, [0] * 4 + [1] * 5])
    seqs = model.generate(ids, attention_mask=mask, max_new_tokens=5).sequences
    assert seqs[0, 9:].tolist() == _greedy(cfg, w, a, 5) and seqs[1, 9:].tolist() == _greedy(cfg, w, b, 5)
    assert model.generate(torch.tensor([a]), max_new_tokens=3, num_beams=2).sequences.shape == (1, 12)


def test_checkpoint_round_trip_and_registry(tmp_path):
    from easydel_b200.infra.factory import registry
    from easydel_b200.modules.auto import AutoEasyDeLConfig
    from easydel_b200.utils.parameters_transformation import internal_to_hf

    cfg, w, model = C.make(tmp_path, "looped", torch.bfloat16, "cpu")
    names = internal_to_hf(model)
    assert set(names) == set(w) and all(torch.equal(names[k].to(w[k].dtype), w[k]) for k in w)
    model.save_pretrained(str(tmp_path / "saved"))
    again = C.load(str(tmp_path / "saved"), torch.bfloat16, "cpu")
    assert again.config.layers == cfg["layers"] and again.config.loop == cfg["loop"]
    for (n, p), (m, q) in zip(model.named_parameters(), again.named_parameters()):
        assert n == m and torch.equal(p, q), n
    assert AutoEasyDeLConfig.from_pretrained(str(tmp_path / "looped")).model_type == "rakevik"
    assert registry.model_type_of({"architecture": "Rakevik"}) == "rakevik"
    with pytest.raises(KeyError):
        registry.model_type_of({"architecture": "nothing known"})
    bad = dict(cfg, layers=[{"type": "other", "mixer": {}, "mlp": None}])
    with pytest.raises(ValueError, match="unknown mixer"):
        registry.get_config("rakevik")(**bad)


def test_cache_layout(tmp_path):
    """Every run of a looped layer has pages and a state of its own; layers with equal head shapes share a pool."""
    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cpu")
    rep = C.replayer(model)
    cache = rep.engine.cache
    assert [g.layers for g in cache.groups] == [[0], [2, 4, 6]] and set(cache.linear) == set(range(8))
    assert cache._k[0].shape[-1] == 48 and cache._v[0].shape[-1] == 24
    info = model.get_operations_cache_info()
    assert info.is_hybrid_model and info.num_attention_layers == 4


def test_trace_command(tmp_path, monkeypatch, capsys):
    import io
    import json
    import sys

    import numpy as np

    from easydel_b200.inference.esurge import trace_run

    cfg, w, _ = C.make(tmp_path, "plain", torch.float32, "cpu")
    toks = C.tokens(12, cfg["vocab"])
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:10], "want": [0, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[10:11], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[11:], "want": [0]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    assert trace_run.main(["--model", str(tmp_path / "plain"), "--dtype", "float32", "--out", str(tmp_path),
                           "--max-tokens", "64"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, w, toks)
    got = np.concatenate([np.fromfile(tmp_path / f"{n}.f32", dtype="<f4") for n in (0, 2)]).reshape(3, -1)
    assert not (tmp_path / "1.f32").exists()
    assert C.error(torch.from_numpy(got), want[[0, 9, 11]]) < TOL


def test_builder_serves_a_checkpoint_folder(tmp_path):
    """The builder behind ``python -m easydel_b200.elarge`` (serve / eval), without a tokenizer in the folder."""
    from easydel_b200.elarge import eLargeModel
    from easydel_b200.inference import SamplingParams

    cfg, w, _ = C.make(tmp_path, "plain", torch.float32, "cpu")
    elm = eLargeModel.from_pretrained(str(tmp_path / "plain")).set_dtype("float32")
    elm.update("loader", device="cpu").set_esurge(max_model_len=128, max_num_seqs=2)
    assert elm.validate() == []
    prompt = C.tokens(7, cfg["vocab"])
    out = elm.build_esurge().generate([prompt], SamplingParams(max_tokens=3, temperature=0.0, ignore_eos=True))
    assert out[0].outputs[0].token_ids == _greedy(cfg, w, prompt, 3)
