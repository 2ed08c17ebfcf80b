"""Ninisun on the CPU path: mechanisms, caches, batches, generation and checkpoints against a plain restatement."""

import math

import ninisun_cases as C
import oracle_ninisun as O
import pytest
import torch

from easydel_b200.ops import rotation, stream

TOL = 3e-5


def _r(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("scaling", [None, C.YARN, {"factor": 3.0, "original": 4096, "fast": 32.0, "slow": 1.0},
                                     {"factor": 2.0, "original": 7, "fast": 32.0, "slow": 1.0},      # the slowest pairs too
                                     {"factor": 2.0, "original": 10 ** 9, "fast": 4.0, "slow": 4.0}])
@pytest.mark.parametrize("base,dims", [(500.0, 16), (1e6, 128), (10.0, 2)])
def test_scaled_frequencies(scaling, base, dims):
    f = rotation.pair_frequencies(base, dims, scaling=scaling).double()
    n = dims // 2
    want = torch.tensor([O.frequency(base, dims, i, scaling) for i in range(n)], dtype=torch.double)
    assert torch.allclose(f[:n] + f[n:], want, rtol=1e-12, atol=0)
    assert rotation.magnitude(scaling) == (0.1 * math.log(scaling["factor"]) + 1 if scaling else 1.0)
    llama = {"factor": 2.0, "low": 1.0, "high": 4.0, "original": 64}
    assert rotation.magnitude(llama) == 1.0


def test_prologue_rows():
    """Biases, rotated neighbours with a magnitude, blended values."""
    H, G, D, V, T = 3, 1, 10, 4, 6
    qkv, bias, first = _r(T, H * D + G * (D + V)), _r(H * D + G * (D + V), seed=1), _r(T, G, V, seed=2)
    pos = torch.tensor([0, 1, 2, 70, 900, 50001])
    rot = {"base": 40.0, "dims": 6, "scaling": C.YARN}
    freq = rotation.pair_frequencies(40.0, 6, scaling=C.YARN)
    q, k, v = stream.rotary_rows(qkv, (H, G, D, V), None, None, 0.0, pos, freq, "neighbours", rotation.magnitude(C.YARN), bias,
                                 first, torch.tensor(0.3))
    row = qkv + bias
    assert torch.allclose(q, O.rotate(row[:, :H * D].view(T, H, D), pos, rot), atol=1e-5)
    assert torch.allclose(k, O.rotate(row[:, H * D:(H + G) * D].view(T, G, D), pos, rot), atol=1e-5)
    assert torch.allclose(v.reshape(T, -1), 0.7 * row[:, (H + G) * D:] + 0.3 * first.flatten(1), atol=1e-6)


def test_kept_first_tokens_and_sigmoid_weights():
    from easydel_b200.ops import reference as R
    from easydel_b200.ops.serving import SigmoidWeights

    assert O.visible(6, 2, 1).tolist() == [[j <= i and (i - j < 2 or j == 0) for j in range(6)] for i in range(6)]
    q, k, v, pb, g = 3 * _r(20, 4, 8), _r(20, 2, 8, seed=1), _r(20, 2, 6, seed=2), _r(4, seed=3), _r(20, 4, seed=4)
    kw = dict(scale=0.7, sliding_window=5, keep_first=3)
    got = R.attention(q[None], k[None], v[None], **kw)[0]
    assert torch.allclose(got, O.softmax_heads(q, k, v, 0.7, 5, 3), atol=1e-5)
    assert not torch.allclose(got, O.softmax_heads(q, k, v, 0.7, 5, 2), atol=1e-2)
    got = R.attention(q[None], k[None], v[None], score_bias=pb, **kw)[0]
    want = O.sigmoid_heads(q, k, v, 0.7, pb, 5, 3)
    assert torch.allclose(got, want, atol=1e-5)
    assert torch.allclose(SigmoidWeights(pb, g, 1.7).finish(got), 1.7 * want * O.sigmoid(g)[..., None], atol=1e-5)


def test_normed_and_scaled_branches():
    x, y, wb, ls, w = _r(9, 12), 5 * _r(9, 12, seed=1), 1 + 0.2 * _r(12, seed=2), _r(12, seed=3), 1 + 0.2 * _r(12, seed=4)
    for scale in (ls, None):
        s, h = stream.add_norm(x, stream.NormedBranch(y, wb, 1e-3, scale), 1.0, w, 1e-5, torch.bfloat16)
        want = x + O.rms_norm(y, wb, 1e-3) * (1.0 if scale is None else scale)
        assert torch.allclose(s, want, atol=1e-5) and torch.equal(h, O.rms_norm(s, w, 1e-5).to(torch.bfloat16))


def test_generalised_delta_rule_over_portions():
    from easydel_b200.ops import ssm

    H, D, V, T, rank = 2, 5, 3, 40, 4
    wt = ssm.DeltaWeights(_r(H * D, rank), _r(H * D, seed=1) - 2, _r(H * D, seed=2), 1 + 0.1 * _r(H * V, seed=3),
                          math.exp(-0.5), 1e-6, 1e-5)
    cols = ssm.DeltaColumns(*(_r(T, n, seed=10 + i) for i, n in enumerate((H * D, H * D, H * V, H * D, H * V, rank))))
    h3 = lambda t: t.view(T, H, -1)  # noqa: E731
    w = torch.exp(-math.exp(-0.5) * O.sigmoid(torch.tanh(cols.x) @ wt.w2.t() + wt.w0))
    o, S = O.delta_rule(h3(cols.r), h3(w), h3(cols.k), h3(O.sigmoid(cols.a + wt.a0)), h3(cols.v))
    o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + 1e-5)).reshape(T, -1) * wt.norm * O.sigmoid(cols.g) * 0.8
    run = lambda c, cu, **kw: ssm.generalized_delta_rule(c, (H, D, V), wt, torch.tensor(cu, dtype=torch.int32),  # noqa: E731
                                                         max(b - a for a, b in zip(cu, cu[1:])), scale=0.8, **kw)
    state = torch.zeros(3, H, D, V)
    assert torch.allclose(run(cols, [0, T], slots=torch.tensor([1]), state=state), o, atol=1e-5)
    assert torch.allclose(state[1], S, atol=1e-5) and not state[0].any() and not state[2].any()
    state.zero_()
    for a, b in ((0, 2), (2, 3), (3, 31), (31, T)):
        part = ssm.DeltaColumns(*(t[a:b] for t in vars(cols).values()))
        out = torch.empty(b - a, H * V)
        assert run(part, [0, b - a], slots=torch.tensor([2]), state=state, out=out) is out
        assert torch.allclose(out, o[a:b], atol=1e-5)
    assert torch.allclose(state[2], S, atol=1e-5)
    two = ssm.DeltaColumns(*(torch.cat([t[:7], t]) for t in vars(cols).values()))
    assert torch.allclose(run(two, [0, 7, 7 + T]), torch.cat([o[:7], o]), atol=1e-5)


# ------------------------------------------------------------------------------------------------ whole models
@pytest.mark.parametrize("name", sorted(C.CONFIGS))
def test_logits_and_hidden_states(tmp_path, name):
    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    toks = C.tokens(150, cfg["vocab"])
    res = []
    want = O.forward(cfg, w, toks, layers=res)
    with torch.no_grad():
        out = model(input_ids=torch.tensor([toks]), output_hidden_states=True)
    assert C.error(out.logits[0], want) < TOL
    assert len(out.hidden_states) == len(cfg["layers"]) + 1
    for a, b in zip(out.hidden_states[1:-1], res):
        assert C.error(a[0], b) < TOL
    toks = toks[:40]
    want = O.forward(cfg, w, toks)
    with torch.enable_grad():      # the differentiable form: no cache, batch of two equal rows
        lg = model(input_ids=torch.tensor([toks, toks[::-1]])).logits
        assert C.error(lg[0], want) < TOL
        assert C.error(lg[1], O.forward(cfg, w, toks[::-1])) < TOL
        lg.square().mean().backward()
    # the first layer that blends values has nothing to blend with
    first = next((i for i, e in enumerate(cfg["layers"]) if e["type"] == "attention" and e["mixer"]["v_mix"]), None)
    idle = {n for n, p in model.named_parameters() if p.grad is None}
    assert idle == {f"model.layers.{i}.self_attn.value_mix" for i in [first] if i is not None}


def test_values_blend_only_where_the_configuration_says(tmp_path):
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
    names = [n for n, _ in model.named_parameters() if n.endswith("value_mix")]
    assert "model.layers.2.self_attn.value_mix" not in names and "model.layers.4.self_attn.value_mix" in names
    cfg2 = O.random_config([O.windowed(2, 2, 8, 4, 0.3, 9, 1), O.windowed(2, 1, 8, 8, 0.3, 9, 1)], 32, 40)
    _, _, bad = C.make(tmp_path, "bad", torch.float32, "cpu", cfg=cfg2)
    with pytest.raises(ValueError, match="cannot blend"), torch.no_grad():
        bad(input_ids=torch.tensor([[1, 2, 3]]))


MUTATIONS = ["no_rotation", "no_scaling", "no_magnitude", "no_mixing", "wide_window", "narrow_window", "keep_more", "keep_fewer",
             "no_bias", "no_score_bias", "softmax", "no_gate", "no_decay", "no_removal", "no_layer_scale"]


def test_a_wrong_mechanism_would_show(tmp_path):
    """The comparison is sharp enough to notice each of these mistakes (planted in the oracle)."""
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
    toks = C.tokens(140, cfg["vocab"])
    with torch.no_grad():
        got = model(input_ids=torch.tensor([toks])).logits[0]
    assert C.error(got, O.forward(cfg, w, toks)) < TOL
    for m in MUTATIONS:
        assert C.error(got, O.forward(cfg, w, toks, mutate=m)) > 100 * TOL, m


@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
@pytest.mark.parametrize("cuts", [[140, 1], [2], [127, 2, 1, 3], [1]])
def test_portions_and_decoding_match_the_whole(tmp_path, name, cuts):
    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    toks = C.tokens(150 if cuts != [1] else 40, cfg["vocab"], 3)
    want = O.forward(cfg, w, toks)
    assert C.error(C.run_cut(C.replayer(model), "a", toks, cuts), want) < TOL


def test_windows_give_pages_back_but_the_first_ones(tmp_path):
    cfg = O.random_config([O.windowed(2, 1, 16, 16, 0.3, 20, 0, mlp=O.dense(32)), O.windowed(2, 1, 16, 16, 0.3, 20, 3),
                           O.windowed(2, 1, 16, 16, 0.3, 140, 129), O.parallel((2, 1, 8, 8, 0.3, 8, 50.0, None), (2, 8))], 40, 50)
    cfg, w, model = C.make(tmp_path, "windows", torch.float32, "cpu", cfg=cfg)
    rep = C.replayer(model, max_tokens=768, max_requests=1)
    assert [(m.bounded, m.kept_pages) for m in rep.engine.kv.managers] == [(False, 0), (True, 0), (True, 1), (True, 2)]
    toks = C.tokens(700, cfg["vocab"])
    got = [C.run_cut(rep, "a", toks[:680], [100, 128, 97], end=False)]
    req = rep.requests["a"]
    for t in toks[680:]:
        got.append(rep.step([{"id": "a", "tokens": [t], "want": [0]}]))
    assert rep.engine.kv.pages_held(req) == [6, 1, 2, 4]
    assert C.error(torch.cat(got), O.forward(cfg, w, toks)) < TOL


def test_page_manager_and_prefix_hits_with_kept_tokens():
    from easydel_b200.caching import specs as SP
    from easydel_b200.inference.esurge.kv_manager import GroupManager
    from easydel_b200.inference.esurge.page_pool import NULL_PAGE

    spec = SP.SlidingWindowSpec(sliding_window=200, keep_first=130)
    assert spec.tokens_kept(1000) == 330 and spec.pages_per_sequence(4096, 1) == 2 + 1 + 2
    assert spec.group_key() != SP.SlidingWindowSpec(sliding_window=200).group_key()
    m = GroupManager(spec, num_pages=32)
    pages = m.pool.allocate(8)
    own = list(pages)
    assert m.remove_skipped(pages, 900) == 3            # keys from 701 on: pages 5 .. 7, and the first two
    assert pages == own[:2] + [NULL_PAGE] * 3 + own[5:]
    assert m.remove_skipped(pages, 900) == 0
    hashes = [bytes([i]) for i in range(8)]
    for i in (0, 1, 5, 6, 7):
        m.pool.register(pages[i], hashes[i])
    assert m.holds(hashes, 8)          # a hit of 8 pages: the next query sits at 1024 and sees keys from 825 on
    assert m.take_cached(hashes, 8) == own[:2] + [NULL_PAGE] * 4 + own[6:]
    m.pool.cached.pop(hashes[1])
    assert not m.holds(hashes, 8)


def test_mixed_batches_reuse_pages_and_slots(tmp_path):
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
    rep = C.replayer(model, max_tokens=512, max_requests=3)
    pool_free = [m.pool.num_free for m in rep.engine.kv.managers]
    seqs = {n: C.tokens(k, cfg["vocab"], i) for i, (n, k) in enumerate(
        [("a", 131), ("b", 5), ("c", 90), ("d", 129), ("e", 2)])}
    plan = [[("a", 60), ("b", 1)], [("a", 70), ("b", 2), ("c", 64)], [("b", 2), ("a", 1)], [("c", 1), ("d", 100)],
            [("d", 2), ("c", 25), ("e", 1)], [("d", 27), ("e", 1)]]
    for n, lg in C.feed(rep, plan, seqs).items():
        assert C.error(lg, O.forward(cfg, w, seqs[n])) < TOL, n
    assert [m.pool.num_free for m in rep.engine.kv.managers] == pool_free


# ------------------------------------------------------------------------------------------------ engine and checkpoints
@pytest.mark.parametrize("name,async_scheduling", [("mixed", False), ("mixed", True), ("windowed", True)])
def test_greedy_generation_through_the_engine(tmp_path, name, async_scheduling):
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    cfg, w, model = C.make(tmp_path, name, torch.float32, "cpu")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (1, 13, 140, 40)]
    # few slots, a small token budget (prompts are cut) and few pages
    eng = eSurge(model, max_model_len=256, max_num_seqs=3, num_pages=5, max_num_batched_tokens=48,
                 async_scheduling=async_scheduling)
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for p, o in zip(prompts, eng.generate(prompts, sp)):
        assert o.outputs[0].token_ids == C.greedy(cfg, w, p, 6)
    # the same prompt again: its full page may come from the prefix cache (of models without a recurrence)
    assert eng.generate([prompts[2]], sp)[0].outputs[0].token_ids == C.greedy(cfg, w, prompts[2], 6)
    sampled = eng.generate([prompts[1]], SamplingParams(max_tokens=5, temperature=0.8, top_k=5, seed=1))
    assert len(sampled[0].outputs[0].token_ids) <= 5


def test_generate_with_padding_and_beams(tmp_path):
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
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

    cfg, w, model = C.make(tmp_path, "odd", torch.bfloat16, "cpu")
    names = internal_to_hf(model)
    assert set(names) == set(w) and all(torch.equal(names[k].to(w[k].dtype), w[k]) for k in w)
    assert model.config.layers[0]["mixer"]["right"]["rank"] == 5        # read off the tensors
    model.save_pretrained(str(tmp_path / "saved"))
    again = C.load(str(tmp_path / "saved"), torch.bfloat16, "cpu")
    assert again.config.layers == model.config.layers and again.config.norm == cfg["norm"]
    for (n, p), (m, q) in zip(model.named_parameters(), again.named_parameters()):
        assert n == m and torch.equal(p, q), n
    assert AutoEasyDeLConfig.from_pretrained(str(tmp_path / "odd")).model_type == "ninisun"
    assert registry.model_type_of({"architecture": "Ninisun"}) == "ninisun"
    cls = registry.get_config("ninisun")
    assert len(cls().layers) == 2
    layers = cfg["layers"]
    with pytest.raises(ValueError, match="unknown mixer"):
        cls(layers=[{**layers[1], "type": "other"}])
    with pytest.raises(ValueError, match="unknown feed-forward"):
        cls(layers=[{**layers[1], "mlp": {"kind": "moe"}}])
    with pytest.raises(ValueError, match="query heads"):
        cls(layers=[{**layers[1], "mixer": {**layers[1]["mixer"], "kv_heads": 2}}])


def test_every_layer_tensor_keeps_its_own_blend_weight(tmp_path):
    """Checkpoints carry a blend weight for layers that never use it; a folder without them loads as well."""
    cfg = O.random_config([O.windowed(2, 2, 8, 4, 0.3, 9, 1, v_mix=False), O.windowed(2, 2, 8, 4, 0.3, 9, 1),
                           O.windowed(2, 2, 8, 4, 0.3, 9, 1)], 32, 40)
    toks = C.tokens(30, 40)
    for drop in ((), ("l0.mix.vmix",)):
        w = {k: v for k, v in O.random_weights(cfg, 3).items() if k not in drop}
        _, _, model = C.make(tmp_path, f"blend{len(drop)}", torch.float32, "cpu", cfg=cfg, weights=w)
        with torch.no_grad():
            got = model(input_ids=torch.tensor([toks])).logits[0]
        assert C.error(got, O.forward(cfg, w, toks)) < TOL


def test_cache_layout(tmp_path):
    """The twin layers' keys in an unbounded pool, windowed layers in pools of their own, one state per slot."""
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
    cache = C.replayer(model).engine.cache
    assert [(g.window, g.spec.first_kept, g.layers) for g in cache.groups] == [
        (0, 0, [1]), (0, 0, [3]), (20, 40, [4]), (33, 5, [0]), (130, 0, [2])]
    assert [k.shape[-1] for k in cache._k] == [32, 24, 64, 48, 16] and [v.shape[-1] for v in cache._v] == [40, 16, 24, 24, 40]
    assert {i: tuple(s.recurrent.shape[1:]) for i, s in cache.linear.items()} == {1: (3, 16, 16), 3: (2, 40, 40)}
    assert all(s.recurrent.dtype == torch.float32 and s.shift is None for s in cache.linear.values())
    info = model.get_operations_cache_info()
    assert info.is_hybrid_model and info.requires_state_management
    assert [l.tokens_kept(1000) for l in info.layers if l.requires_kv_cache] == [38, 1000, 130, 1000, 60]


def test_trace_command(tmp_path, monkeypatch, capsys):
    import io
    import json
    import sys

    import numpy as np

    from easydel_b200.inference.esurge import trace_run

    cfg, w, _ = C.make(tmp_path, "twin", torch.float32, "cpu")
    toks = C.tokens(12, cfg["vocab"])
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:10], "want": [0, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[10:], "want": [1]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    assert trace_run.main(["--model", str(tmp_path / "twin"), "--dtype", "float32", "--out", str(tmp_path),
                           "--max-tokens", "64"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1"]
    got = np.concatenate([np.fromfile(tmp_path / f"{n}.f32", dtype="<f4") for n in (0, 1)]).reshape(3, -1)
    assert C.error(torch.from_numpy(got), O.forward(cfg, w, toks)[[0, 9, 11]]) < TOL


def test_builder_serves_a_checkpoint_folder(tmp_path):
    """The builder behind ``python -m easydel_b200.elarge`` (serve / eval), without a tokenizer in the folder."""
    from easydel_b200.elarge import eLargeModel
    from easydel_b200.inference import SamplingParams

    cfg, w, _ = C.make(tmp_path, "mixed", torch.float32, "cpu")
    elm = eLargeModel.from_pretrained(str(tmp_path / "mixed")).set_dtype("float32")
    elm.update("loader", device="cpu").set_esurge(max_model_len=128, max_num_seqs=2)
    assert elm.validate() == []
    prompt = C.tokens(7, cfg["vocab"])
    out = elm.build_esurge().generate([prompt], SamplingParams(max_tokens=3, temperature=0.0, ignore_eos=True))
    assert out[0].outputs[0].token_ids == C.greedy(cfg, w, prompt, 3)
