"""Disunex against a plain restatement of its equations, on the CPU path: mechanisms, caches, batches, generation."""

import disunex_cases as C
import oracle_disunex as O
import pytest
import torch

from easydel_b200.ops import latent, rotation, stream

TOL = 2e-5


def _r(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
def test_norm_after_the_sum():
    x, y, w = _r(9, 12), _r(9, 12, seed=1), 0.2 * _r(12, seed=2)
    s, h = stream.post_norm(x, y, 2.5, w, 1e-5, torch.bfloat16, 1.0)
    want = O.norm_after_sum(x, y, 2.5, w, 1e-5)
    assert torch.allclose(s, want, atol=1e-6) and torch.equal(h, s.to(torch.bfloat16))
    assert torch.allclose(stream.norm_shift(x, w, 1e-5, torch.float32, offset=1.0), O.rms_norm(x, 1 + w, 1e-5), atol=1e-6)


def test_rotation_of_neighbouring_pairs():
    x = _r(7, 3, 10)
    pos = torch.tensor([0, 1, 2, 50, 999, 70001, 5])
    for dims in (10, 4):
        got = rotation.rotate(x, pos, rotation.pair_frequencies(300.0, dims))
        assert torch.allclose(got, O.rotate_pairs(x, pos, 300.0, dims), atol=1e-6)
        assert torch.equal(got[..., dims:], x[..., dims:]) and torch.equal(got[0], x[0])
    # scores depend on the distance only
    q, k = _r(1, 1, 8).expand(6, 1, 8), _r(1, 1, 8, seed=1).expand(6, 1, 8)
    f = rotation.pair_frequencies(50.0, 8)
    p = torch.arange(6) * 3
    a, b = rotation.rotate(q, p + 4, f), rotation.rotate(k, p, f)
    assert torch.allclose((a * b).sum(-1), (a * b).sum(-1)[:1].expand(6, 1), atol=1e-5)


def test_expansion_weight_rebuilds_keys_and_values():
    H, D, R, V, L = 3, 6, 4, 5, 7
    up, rows = _r(H * D + H * V, L), _r(11, L + R, seed=1)
    kv = rows @ latent.expansion_weight(up, H, D, R, V, L).T
    k = kv[:, :H * (D + R)].view(11, H, D + R)
    for h in range(H):
        assert torch.allclose(k[:, h, :D], rows[:, :L] @ up[h * D:(h + 1) * D].T, atol=1e-5)
        assert torch.equal(k[:, h, D:], rows[:, L:])
    assert torch.allclose(kv[:, H * (D + R):], rows[:, :L] @ up[H * D:].T, atol=1e-5)


def test_window_mask_and_sink():
    assert O.visible(5, 2).tolist() == [[i - 2 < j <= i for j in range(5)] for i in range(5)]
    s, sink = _r(4, 6), torch.tensor([0.7])
    p = O.sink_softmax(s, sink)
    full = torch.softmax(torch.cat([s, sink.expand(4, 1)], 1), 1)
    assert torch.allclose(p, full[:, :-1], atol=1e-6) and bool((p.sum(1) < 1).all())


def test_routing_and_clamped_experts():
    from easydel_b200.layers.moe import MoEBlock

    torch.manual_seed(0)
    blk = MoEBlock(12, 7, 5, 2, scoring="sigmoid", use_score_bias=True, act_limit=0.4, expert_init_std=0.5, init_std=0.5)
    with torch.no_grad():
        blk.e_score_correction_bias.copy_(torch.tensor([0.0, 0.9, -0.5, 0.2, 0.1]))
    h = 2 * _r(30, 12)
    w = {"m.router": blk.gate.weight, "m.correction": blk.e_score_correction_bias}
    for e in range(5):
        w.update({f"m.e{e}.gate": blk.gate_up_proj.weight[e, :7], f"m.e{e}.up": blk.gate_up_proj.weight[e, 7:],
                  f"m.e{e}.down": blk.down_proj.weight[e]})
    spec = O.experts(5, 2, 7, 0.4)
    with torch.no_grad():
        got = blk.stream_rows(h)
        assert torch.allclose(got, O.moe(h, w, "m", spec), atol=1e-5)
        for m in ("no_correction", "corrected_weights"):
            assert not torch.allclose(got, O.moe(h, w, "m", spec, m), atol=1e-3)
        assert not torch.allclose(got, O.moe(h, w, "m", O.experts(5, 2, 7, 0.5)), atol=1e-3)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_logits_and_hidden_states(tmp_path, name):
    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    toks = C.tokens(150, cfg["vocab"])
    res = []
    want = O.forward(cfg, w, toks, residuals=res)
    with torch.no_grad():
        out = model(input_ids=torch.tensor([toks]), output_hidden_states=True)
    assert C.error(out.logits[0], want) < TOL
    assert len(out.hidden_states) == len(cfg["layers"]) + 1
    for a, b in zip(out.hidden_states[1:-1], res):
        assert C.error(a[0], b) < TOL
    last = O.rms_norm(res[-1], 1 + w["final.norm"].double(), cfg["norm"]["eps"])
    assert C.error(out.hidden_states[-1][0], last) < TOL
    with torch.enable_grad():      # the differentiable form: no cache, batch of two equal rows
        lg = model(input_ids=torch.tensor([toks, toks[::-1]])).logits
        assert C.error(lg[0], want) < TOL
        assert C.error(lg[1], O.forward(cfg, w, toks[::-1])) < TOL
        lg.square().mean().backward()
    # the correction only steers the choice, so it has no gradient
    assert all(p.grad is not None for n, p in model.named_parameters() if "correction" not in n)


@pytest.mark.parametrize("mutate", ["no_sink", "scaled_sink", "window_plus", "window_minus", "no_rotation", "no_gate",
                                    "no_alpha", "no_correction", "corrected_weights"])
def test_a_wrong_mechanism_would_show(tmp_path, mutate):
    """The comparison is sharp enough to notice each of these mistakes (planted in the oracle)."""
    cfg, w, model = C.make(tmp_path, "shared", torch.float32, "cpu")
    toks = C.tokens(140, cfg["vocab"])
    with torch.no_grad():
        got = model(input_ids=torch.tensor([toks])).logits[0]
    assert C.error(got, O.forward(cfg, w, toks)) < TOL
    assert C.error(got, O.forward(cfg, w, toks, mutate=mutate)) > 100 * TOL


@pytest.mark.parametrize("name", ["shared", "odd", "wide"])
@pytest.mark.parametrize("cuts", [[140, 1], [2], [127, 2, 1, 3], [1]])
def test_portions_and_decoding_match_the_whole(tmp_path, name, cuts):
    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    toks = C.tokens(150 if cuts != [1] else 40, cfg["vocab"], 3)
    want = O.forward(cfg, w, toks)
    assert C.error(C.run_cut(C.replayer(model), "a", toks, cuts), want) < TOL


def test_windows_give_pages_back(tmp_path):
    """A long sequence holds the pages of its windows only, and a pool of that size is enough for it."""
    cfg = O.random_config([O.latent(2, 16, 8, 16, 24, 0.3, window=20, mlp=O.dense(32)),
                           O.latent(2, 16, 8, 16, 24, 0.3, window=140)], 40, 50)
    cfg, w, model = C.make(tmp_path, "windows", torch.float32, "cpu", cfg=cfg)
    rep = C.replayer(model, max_tokens=640, max_requests=1)
    assert [m.bounded for m in rep.engine.kv.managers] == [True, True]
    toks = C.tokens(600, cfg["vocab"])
    got = [C.run_cut(rep, "a", toks[:580], [100, 128, 97], end=False)]
    req = rep.requests["a"]
    held = []
    for t in toks[580:]:
        got.append(rep.step([{"id": "a", "tokens": [t], "want": [0]}]))
        held.append(rep.engine.kv.pages_held(req))
    assert held[-1] == [1, 2]
    assert C.error(torch.cat(got), O.forward(cfg, w, toks)) < TOL


def test_mixed_batches_reuse_pages(tmp_path):
    cfg, w, model = C.make(tmp_path, "shared", torch.float32, "cpu")
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


# ------------------------------------------------------------------------------------------------ engine and checkpoints
@pytest.mark.parametrize("async_scheduling", [False, True])
def test_greedy_generation_through_the_engine(tmp_path, async_scheduling):
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    cfg, w, model = C.make(tmp_path, "shared", torch.float32, "cpu")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (1, 13, 140, 40)]
    # few slots, a small token budget (prompts are cut) and few pages
    eng = eSurge(model, max_model_len=256, max_num_seqs=3, num_pages=4, max_num_batched_tokens=48,
                 async_scheduling=async_scheduling)
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for p, o in zip(prompts, eng.generate(prompts, sp)):
        assert o.outputs[0].token_ids == C.greedy(cfg, w, p, 6)
    # the same prompt again: its full page may come from the prefix cache
    assert eng.generate([prompts[2]], sp)[0].outputs[0].token_ids == C.greedy(cfg, w, prompts[2], 6)
    sampled = eng.generate([prompts[1]], SamplingParams(max_tokens=5, temperature=0.8, top_k=5, seed=1))
    assert len(sampled[0].outputs[0].token_ids) <= 5


def test_generate_with_padding_and_beams(tmp_path):
    cfg, w, model = C.make(tmp_path, "shared", torch.float32, "cpu")
    a, b = C.tokens(9, cfg["vocab"], 1), C.tokens(5, cfg["vocab"], 2)
    ids = torch.tensor([a, [0] * 4 + b])
    mask = torch.tensor([[1] * 9, [0] * 4 + [1] * 5])
    seqs = model.generate(ids, attention_mask=mask, max_new_tokens=5).sequences
    assert seqs[0, 9:].tolist() == C.greedy(cfg, w, a, 5) and seqs[1, 9:].tolist() == C.greedy(cfg, w, b, 5)
    assert model.generate(torch.tensor([a]), max_new_tokens=3, num_beams=2).sequences.shape == (1, 12)


def test_checkpoint_round_trip_and_registry(tmp_path):
    from easydel_b200.infra.factory import registry
    from easydel_b200.modules.auto import AutoEasyDeLConfig
    from easydel_b200.utils.parameters_transformation import internal_to_hf

    cfg, w, model = C.make(tmp_path, "shared", torch.bfloat16, "cpu")
    names = internal_to_hf(model)
    assert set(names) == set(w) and all(torch.equal(names[k].to(w[k].dtype), w[k]) for k in w)
    assert len(model.model.layers) == 3 and model.model.layer_runs == [0, 1, 2, 1, 0, 2]
    model.save_pretrained(str(tmp_path / "saved"))
    again = C.load(str(tmp_path / "saved"), torch.bfloat16, "cpu")
    assert again.config.layers == cfg["layers"] and again.config.postln_alpha == cfg["postln_alpha"]
    for (n, p), (m, q) in zip(model.named_parameters(), again.named_parameters()):
        assert n == m and torch.equal(p, q), n
    assert AutoEasyDeLConfig.from_pretrained(str(tmp_path / "shared")).model_type == "disunex"
    assert registry.model_type_of({"architecture": "Disunex"}) == "disunex"
    cls = registry.get_config("disunex")
    layers = cfg["layers"]
    with pytest.raises(ValueError, match="unknown mixer"):
        cls(layers=[{**layers[0], "type": "other"}])
    with pytest.raises(ValueError, match="unknown feed-forward"):
        cls(layers=[{**layers[0], "mlp": {"kind": "other"}}])
    with pytest.raises(ValueError, match="does not exist"):
        cls(layers=[{**layers[0], "weights_of": 4}])
    with pytest.raises(ValueError, match="nobody's own"):
        cls(layers=[{**layers[0], "weights_of": 1}, {**layers[0], "weights_of": 0}])
    assert cls(layers=[layers[0], {**layers[0], "weights_of": 0}, {**layers[0], "weights_of": 1}]).weight_layers() == \
        ([0], [0, 0, 0])


def test_weights_may_belong_to_a_later_layer(tmp_path):
    layers = [O.latent(2, 16, 8, 16, 24, 0.3, window=9, mlp=O.dense(32)), O.latent(3, 8, 4, 8, 16, 0.3, window=30)]
    cfg = O.random_config([O.again(layers, 1), layers[1], layers[0], O.again(layers, 0)], 40, 50)
    cfg["layers"][0]["weights_of"], cfg["layers"][3]["weights_of"] = 1, 2
    cfg, w, model = C.make(tmp_path, "later", torch.float32, "cpu", cfg=cfg)
    toks = C.tokens(60, 50)
    assert model.model.layer_runs == [0, 0, 1, 1]
    assert C.error(C.run_cut(C.replayer(model), "a", toks, [33, 1, 2]), O.forward(cfg, w, toks)) < TOL


def test_cache_layout(tmp_path):
    """Every run of a layer has pages of its own; runs with the same window and row width share a pool's page table."""
    cfg, w, model = C.make(tmp_path, "shared", torch.float32, "cpu")
    rep = C.replayer(model)
    cache = rep.engine.cache
    assert [(g.window, g.layers) for g in cache.groups] == [(33, [0, 2, 4, 5]), (130, [1, 3])]
    assert cache.latent and not cache.linear and cache._k[0].shape[-1] == 80 and cache._k[1].shape[-1] == 48
    assert all(k is v for k, v in zip(cache._k, cache._v))
    assert cache.groups[1].spec.page_size_bytes == 128 * 48 * 4
    info = model.get_operations_cache_info()
    assert not info.is_hybrid_model and info.num_attention_layers == 6
    assert [l.tokens_kept(1000) for l in info.layers] == [33, 130, 33, 130, 33, 33]


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
    assert out[0].outputs[0].token_ids == C.greedy(cfg, w, prompt, 3)
