"""Gasetar against a plain restatement of its equations, on the CPU path: mechanisms, caches, batches, generation."""

import gasetar_cases as C
import oracle_gasetar as O
import pytest
import torch

from easydel_b200.ops import rotation, stream

TOL = 2e-5


def _r(*s, seed=0):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ------------------------------------------------------------------------------------------------ mechanisms
@pytest.mark.parametrize("scaling", [None, (4.0, 1.0, 4.0, 200), (2.5, 0.5, 16.0, 1000)])
def test_rotation_of_halves_and_its_frequencies(scaling):
    rot = {"base": 700.0, "dims": 12}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    f = rotation.pair_frequencies(rot["base"], rot["dims"], None, rot.get("scaling"))
    want = torch.tensor([O.frequency(700.0, 12, i, rot.get("scaling")) for i in range(6)], dtype=torch.float64)
    assert torch.allclose(f[:6].double() + f[6:].double(), want, rtol=1e-13)
    if scaling and scaling[0] == 4.0:      # every band of the scaling takes part
        plain = torch.tensor([O.frequency(700.0, 12, i) for i in range(6)], dtype=torch.float64)
        ratio = (want / plain).tolist()
        assert 1.0 in ratio and 0.25 in ratio and any(0.26 < r < 0.99 for r in ratio)
    x = _r(7, 3, 16)
    pos = torch.tensor([0, 1, 2, 50, 999, 70001, 5])
    got = rotation.rotate(x, pos, f, "halves")
    assert torch.allclose(got, O.rotate_half(x, pos, rot), atol=1e-6)
    assert torch.equal(got[..., 12:], x[..., 12:]) and torch.equal(got[0], x[0])
    # scores depend on the distance only
    q, k = _r(1, 1, 12).expand(6, 1, 12), _r(1, 1, 12, seed=1).expand(6, 1, 12)
    p = torch.arange(6) * 3
    s = (rotation.rotate(q, p + 4, f, "halves") * rotation.rotate(k, p, f, "halves")).sum(-1)
    assert torch.allclose(s, s[:1].expand(6, 1), atol=1e-5)
    with pytest.raises(ValueError):
        rotation.check_rotation(5, 8, "halves")
    with pytest.raises(ValueError):
        rotation.check_rotation(4, 8, "thirds")


def test_tables_use_the_same_scaling():
    from easydel_b200.layers.rotary import RopeConfig, get_inv_frequencies

    cfg = RopeConfig("llama3", factor=4.0, low_freq_factor=1.0, high_freq_factor=4.0, original_max_position_embeddings=200)
    inv, _ = get_inv_frequencies(cfg, 700.0, 12, 4096)
    s = dict(zip(("factor", "low", "high", "original"), (4.0, 1.0, 4.0, 200)))
    assert torch.allclose(inv, torch.tensor([O.frequency(700.0, 12, i, s) for i in range(6)]), rtol=1e-5)


def test_norms_over_the_whole_projection_then_rotation():
    H, G, D = 3, 2, 8
    q, k, qw, kw = _r(5, H * D), _r(5, G * D, seed=1), _r(H * D, seed=2), _r(G * D, seed=3)
    rot = {"base": 50.0, "dims": 6}
    pos = torch.tensor([0, 3, 4, 5, 90])
    a, b = stream.qk_norm_rotate(q, k, D, qw, kw, 1e-4, pos, rotation.pair_frequencies(50.0, 6))
    assert torch.allclose(a, O.rotate_half(O.rms_norm(q, qw, 1e-4).view(5, H, D), pos, rot), atol=1e-6)
    assert torch.allclose(b, O.rotate_half(O.rms_norm(k, kw, 1e-4).view(5, G, D), pos, rot), atol=1e-6)


def test_window_cap_and_sink():
    from easydel_b200.ops import reference as R

    assert O.visible(5, 2).tolist() == [[i - 2 < j <= i for j in range(5)] for i in range(5)]
    q, k, v = 3 * _r(20, 4, 8), _r(20, 2, 8, seed=1), _r(20, 2, 6, seed=2)
    want = O.windowed_heads(q, k, v, 0.7, 5, 2.0)
    got = R.attention(q[None], k[None], v[None], scale=0.7, sliding_window=5, softcap=2.0)[0]
    assert torch.allclose(got, want, atol=1e-5)
    assert not torch.allclose(got, O.windowed_heads(q, k, v, 0.7, 5, 0.0), atol=1e-2)
    s, sink = _r(4, 6), torch.tensor([0.7])
    p = O.sink_softmax(s, sink)
    assert torch.allclose(p, torch.softmax(torch.cat([s, sink.expand(4, 1)], 1), 1)[:, :-1], atol=1e-6)


def test_sum_and_norm_and_capped_logits():
    from easydel_b200.ops.moe_kernels import ExpertRows

    x, y, w = _r(9, 12), _r(9, 12, seed=1), 1 + 0.2 * _r(12, seed=2)
    s, h = stream.add_norm(x, y, 0.3, w, 1e-5, torch.bfloat16)
    assert torch.allclose(s, x + 0.3 * y) and torch.equal(h, O.rms_norm(s, w, 1e-5).to(torch.bfloat16))
    s, h = stream.add_norm(x, None, 0.3, w, 1e-5, torch.float32)
    assert s is x and torch.allclose(h, O.rms_norm(x, w, 1e-5), atol=1e-6)
    ys, wts, pos = _r(20, 12, seed=3), torch.rand(9, 2), torch.randint(0, 20, (18,), dtype=torch.int32)
    rows = ExpertRows(ys, wts, pos, y)
    s, _ = stream.add_norm(x, rows, 2.0, w, 1e-5, torch.float32)
    assert torch.allclose(s, x + 2.0 * (y + (ys[pos.long()].view(9, 2, 12) * wts[..., None]).sum(1)), atol=1e-5)
    z = 5 * _r(4, 7)
    assert torch.allclose(stream.scale_cap(z, 0.4, 1.5), O.soft_cap(0.4 * z, 1.5), atol=1e-6)
    assert torch.allclose(stream.scale_cap(z, 0.4), 0.4 * z)


def test_routing_and_experts():
    from easydel_b200.layers.moe import MoEBlock

    torch.manual_seed(0)
    blk = MoEBlock(12, 7, 5, 2, scoring="softmax", router_bias=True, shared_intermediate_size=9, expert_init_std=0.5,
                   init_std=0.5)
    with torch.no_grad():
        blk.gate.bias.copy_(torch.tensor([0.0, 0.9, -0.5, 0.2, 0.1]))
    h, base = 2 * _r(30, 12), _r(30, 12, seed=5)
    sh = blk.shared_experts
    w = {"m.router": blk.gate.weight, "m.router.b": blk.gate.bias, "m.shared.gate": sh.gate_up_proj.weight[:9],
         "m.shared.up": sh.gate_up_proj.weight[9:], "m.shared.down": sh.down_proj.weight}
    for e in range(5):
        w.update({f"m.e{e}.gate": blk.gate_up_proj.weight[e, :7], f"m.e{e}.up": blk.gate_up_proj.weight[e, 7:],
                  f"m.e{e}.down": blk.down_proj.weight[e]})
    spec = O.experts(5, 2, 7, 9)
    with torch.no_grad():
        got = blk.stream_rows(h)
        assert torch.allclose(got, O.moe(h, w, "m", spec), atol=1e-5)
        assert torch.allclose(blk.stream_rows(h, base.clone()), got + base, atol=1e-5)
        for m in ("no_router_bias", "softmax_over_all", "no_shared"):
            assert not torch.allclose(got, O.moe(h, w, "m", spec, m), atol=1e-3)


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
    last = O.rms_norm(res[-1], w["final.norm"].double(), cfg["norm"]["eps"])
    assert C.error(out.hidden_states[-1][0], last) < TOL
    with torch.enable_grad():      # the differentiable form: no cache, batch of two equal rows
        lg = model(input_ids=torch.tensor([toks, toks[::-1]])).logits
        assert C.error(lg[0], want) < TOL
        assert C.error(lg[1], O.forward(cfg, w, toks[::-1])) < TOL
        lg.square().mean().backward()
    assert all(p.grad is not None for p in model.parameters())


MUTATIONS = ["no_sink", "scaled_sink", "window_plus", "window_minus", "no_rotation", "neighbour_pairs", "no_scaling",
             "head_norms", "wrong_groups", "no_score_cap", "no_gate", "no_router_bias", "softmax_over_all", "no_shared",
             "one_after_the_other", "no_residual_mult", "no_logit_scale", "no_logit_cap"]


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


def test_windows_give_pages_back(tmp_path):
    """A long sequence holds every page of its latents and the pages of its windows only."""
    cfg = O.random_config([O.windowed(2, 1, 16, 16, 0.3, 20, 5.0, mlp=O.dense(32)), O.latent(2, 16, 8, 16, 24, 0.3),
                           O.windowed(2, 1, 16, 16, 0.3, 140, 5.0)], 40, 50)
    cfg, w, model = C.make(tmp_path, "windows", torch.float32, "cpu", cfg=cfg)
    rep = C.replayer(model, max_tokens=640, max_requests=1)
    assert [m.bounded for m in rep.engine.kv.managers] == [False, True, True]
    toks = C.tokens(600, cfg["vocab"])
    got = [C.run_cut(rep, "a", toks[:580], [100, 128, 97], end=False)]
    req = rep.requests["a"]
    held = []
    for t in toks[580:]:
        got.append(rep.step([{"id": "a", "tokens": [t], "want": [0]}]))
        held.append(rep.engine.kv.pages_held(req))
    assert held[-1] == [5, 1, 2]
    assert C.error(torch.cat(got), O.forward(cfg, w, toks)) < TOL


def test_mixed_batches_reuse_pages(tmp_path):
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
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

    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (1, 13, 140, 40)]
    # few slots, a small token budget (prompts are cut) and few pages
    eng = eSurge(model, max_model_len=256, max_num_seqs=3, num_pages=5, max_num_batched_tokens=48,
                 async_scheduling=async_scheduling)
    sp = SamplingParams(max_tokens=6, temperature=0.0, ignore_eos=True)
    for p, o in zip(prompts, eng.generate(prompts, sp)):
        assert o.outputs[0].token_ids == C.greedy(cfg, w, p, 6)
    # the same prompt again: its full page may come from the prefix cache
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


def test_training_loss_sees_the_logit_scale_and_cap(tmp_path):
    cfg, w, model = C.make(tmp_path, "windowed", torch.float32, "cpu")
    toks = C.tokens(30, cfg["vocab"])
    lg = O.forward(cfg, w, toks)
    want = torch.nn.functional.cross_entropy(lg[:-1], torch.tensor(toks[1:]))
    ids = torch.tensor([toks])
    _, metrics = model.compute_loss(input_ids=ids, labels=ids)
    assert abs(float(metrics.loss) - float(want)) < 1e-4


def test_checkpoint_round_trip_and_registry(tmp_path):
    from easydel_b200.infra.factory import registry
    from easydel_b200.modules.auto import AutoEasyDeLConfig
    from easydel_b200.utils.parameters_transformation import internal_to_hf

    cfg, w, model = C.make(tmp_path, "mixed", torch.bfloat16, "cpu")
    names = internal_to_hf(model)
    assert set(names) == set(w) and all(torch.equal(names[k].to(w[k].dtype), w[k]) for k in w)
    model.save_pretrained(str(tmp_path / "saved"))
    again = C.load(str(tmp_path / "saved"), torch.bfloat16, "cpu")
    for key in ("layers", "embedding", "residual_mult", "logit_scale", "logit_softcap", "norm"):
        assert getattr(again.config, key) == cfg[key], key
    for (n, p), (m, q) in zip(model.named_parameters(), again.named_parameters()):
        assert n == m and torch.equal(p, q), n
    assert AutoEasyDeLConfig.from_pretrained(str(tmp_path / "mixed")).model_type == "gasetar"
    assert registry.model_type_of({"architecture": "Gasetar"}) == "gasetar"
    cls = registry.get_config("gasetar")
    layers = cfg["layers"]
    with pytest.raises(ValueError, match="unknown mixer"):
        cls(layers=[{**layers[0], "type": "other"}])
    with pytest.raises(ValueError, match="unknown feed-forward"):
        cls(layers=[{**layers[0], "mlp": {"kind": "other"}}])
    with pytest.raises(ValueError, match="query heads"):
        cls(layers=[{**layers[0], "mixer": {**layers[0]["mixer"], "kv_heads": 4}}])
    with pytest.raises(ValueError, match="experts"):
        cls(layers=[{**layers[0], "mlp": O.experts(4, 5, 8)}])


def test_cache_layout(tmp_path):
    """Latent rows in an unbounded pool, windowed layers in pools of their own; values may have another width."""
    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cpu")
    cache = C.replayer(model).engine.cache
    assert [(g.spec.latent, g.window, g.layers) for g in cache.groups] == [
        (True, 0, [1]), (True, 0, [3]), (False, 33, [0]), (False, 130, [2])]
    assert [k.shape[-1] for k in cache._k] == [80, 48, 48, 16] and [v.shape[-1] for v in cache._v[2:]] == [24, 40]
    assert cache.groups[2].spec.page_size_bytes == 128 * 2 * (48 + 24) * 4
    info = model.get_operations_cache_info()
    assert not info.is_hybrid_model and [l.tokens_kept(1000) for l in info.layers] == [33, 1000, 130, 1000]


def test_trace_command(tmp_path, monkeypatch, capsys):
    import io
    import json
    import sys

    import numpy as np

    from easydel_b200.inference.esurge import trace_run

    cfg, w, _ = C.make(tmp_path, "windowed", torch.float32, "cpu")
    toks = C.tokens(12, cfg["vocab"])
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:10], "want": [0, 9]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[10:11], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[11:], "want": [0]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("".join(json.dumps(x) + "\n" for x in lines)))
    assert trace_run.main(["--model", str(tmp_path / "windowed"), "--dtype", "float32", "--out", str(tmp_path),
                           "--max-tokens", "64"]) == 0
    assert [x for x in capsys.readouterr().out.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, w, toks)
    got = np.concatenate([np.fromfile(tmp_path / f"{n}.f32", dtype="<f4") for n in (0, 2)]).reshape(3, -1)
    assert C.error(torch.from_numpy(got), want[[0, 9, 11]]) < TOL


def test_builder_serves_a_checkpoint_folder(tmp_path):
    """The builder behind ``python -m easydel_b200.elarge`` (serve / eval), without a tokenizer in the folder."""
    from easydel_b200.elarge import eLargeModel
    from easydel_b200.inference import SamplingParams

    cfg, w, _ = C.make(tmp_path, "latent", torch.float32, "cpu")
    elm = eLargeModel.from_pretrained(str(tmp_path / "latent")).set_dtype("float32")
    elm.update("loader", device="cpu").set_esurge(max_model_len=128, max_num_seqs=2)
    assert elm.validate() == []
    prompt = C.tokens(7, cfg["vocab"])
    out = elm.build_esurge().generate([prompt], SamplingParams(max_tokens=3, temperature=0.0, ignore_eos=True))
    assert out[0].outputs[0].token_ids == C.greedy(cfg, w, prompt, 3)
