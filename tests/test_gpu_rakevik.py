"""Rakevik on the GPU: every kernel of the family against fp32 forms, whole models against a plain restatement."""

import math

import oracle_rakevik as O
import pytest
import rakevik_cases as C
import torch

pytestmark = pytest.mark.gpu

DT = [torch.float32, torch.bfloat16]


@pytest.fixture(autouse=True)
def _no_grad():
    with torch.no_grad():
        yield


def _r(*s, seed=0, dtype=torch.float32):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed)).to(dtype).cuda()


def _i32(*v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def _close(got, want, dtype, scale=1.0):
    tol = 3e-6 if dtype == torch.float32 else 8e-3
    d = (got.double() - want.double()).abs().max() / want.double().abs().max().clamp_min(1e-6)
    assert float(d) < tol * scale, float(d)


# ------------------------------------------------------------------------------------------------ kernels of the stream
@pytest.mark.parametrize("W", [60, 77, 352, 1024, 3000, 8192, 9000])
@pytest.mark.parametrize("dtype", DT)
def test_norm_shift(W, dtype):
    from easydel_b200.ops import stream

    lens = [1, 5, 2, 130]
    cu = _i32(0, 1, 6, 8, 138)
    x, w, mu = 3 * _r(138, W), 1 + 0.1 * _r(W, seed=1), torch.rand(W).cuda()
    slots = _i32(4, 0, 2, 1)
    state = _r(6, W, seed=2)
    ref_state = state.clone()
    want = torch.cat([O.token_shift(torch.cat([ref_state[s:s + 1], O.rms_norm(c, w, 1e-5)]), mu)[1:]
                      for s, c in zip(slots.tolist(), torch.split(x, lens))])
    for s, c in zip(slots.tolist(), torch.split(x, lens)):
        ref_state[s] = O.rms_norm(c, w, 1e-5)[-1]
    got = stream.norm_shift(x, w, 1e-5, dtype, mu, cu, slots, state)
    _close(got, want, dtype)
    _close(state, ref_state, torch.float32)
    _close(stream.norm_shift(x, w, 1e-5, dtype), O.rms_norm(x, w, 1e-5), dtype)
    first = stream.norm_shift(x, w, 1e-5, dtype, mu, cu)        # without a state every sequence starts from zeros
    _close(first[1:6], O.token_shift(O.rms_norm(x[1:6], w, 1e-5), mu), dtype)


@pytest.mark.parametrize("W", [352, 1536, 4096])
@pytest.mark.parametrize("dtype", DT)
def test_norm_shift_over_many_rows(W, dtype):
    """Enough rows for the form that walks several rows per CTA: sequence bounds in every place of such a group."""
    from easydel_b200.ops import stream

    lens = [1, 1, 2, 3, 4, 5, 6, 7, 8, 9, 1, 15, 1000, 1, 1500, 17]
    cu = _i32(*torch.tensor([0, *lens]).cumsum(0).tolist())
    x, w, mu = 3 * _r(sum(lens), W), 1 + 0.1 * _r(W, seed=1), torch.rand(W).cuda()
    slots = torch.randperm(len(lens)).to(torch.int32).cuda()
    state = _r(len(lens), W, seed=2)
    want, ends = [], state.clone()
    for s, c in zip(slots.tolist(), torch.split(x, lens)):
        h = O.rms_norm(c, w, 1e-5)
        want.append(O.token_shift(torch.cat([state[s:s + 1], h]), mu)[1:])
        ends[s] = h[-1]
    _close(stream.norm_shift(x, w, 1e-5, dtype, mu, cu, slots, state), torch.cat(want), dtype)
    _close(state, ends, torch.float32)
    _close(stream.norm_shift(x, w, 1e-5, dtype), O.rms_norm(x, w, 1e-5), dtype)


@pytest.mark.parametrize("dtype", DT)
def test_embedding_operand_and_activation(dtype):
    from easydel_b200.ops import stream

    for W in (40, 33):
        table, ids = _r(50, W, dtype=dtype), torch.randint(0, 50, (19,)).cuda()
        operand = torch.zeros(19, 2 * W, dtype=dtype, device="cuda")
        x = stream.embed(table, ids, operand[:, W:])
        assert torch.equal(x, table[ids].float()) and torch.equal(operand[:, W:], table[ids])
        stream.cast_rows(x * 2, operand[:, :W])
        assert torch.equal(operand[:, :W], (x * 2).to(dtype))
    z, act = 4 * _r(37, 41, dtype=dtype), torch.tensor([0.7, -1.3]).cuda()
    _close(stream.xielu(z, act), O.xielu(z.float(), act), dtype)
    o, w = _r(11, 3, 50), 1 + 0.1 * _r(50, seed=3)
    _close(stream.head_norm(o, w, 1e-4, dtype), O.rms_norm(o, w, 1e-4), dtype)


@pytest.mark.parametrize("M,N,K", [(5, 352, 224), (300, 96, 640), (4, 64, 2048), (7, 53, 60)])
@pytest.mark.parametrize("dtype", DT)
def test_products_accumulate_into_the_stream(M, N, K, dtype):
    """Plain and split-K products with fp32 results and fp32 accumulation."""
    from easydel_b200.ops import stream

    x, w = _r(M, K, dtype=dtype), _r(N, K, seed=1, dtype=dtype) / math.sqrt(K)
    s = 10 * _r(M, N, seed=2)
    want = x.double() @ w.double().t()
    _close(stream.linear_add_(s.clone(), x, w), s.double() + want, torch.float32)
    b = _r(N, seed=4, dtype=dtype)
    _close(stream.linear(x, w, b, torch.float32), want + b.double(), torch.float32, 2)


@pytest.mark.parametrize("heads", [(6, 2, 48, 24), (4, 4, 64, 88), (3, 1, 20, 12), (2, 2, 128, 128), (5, 1, 9, 7)])
@pytest.mark.parametrize("dtype", DT)
def test_attention_prologue(heads, dtype):
    from easydel_b200.ops import stream

    Hq, Hkv, D, Dv = heads
    T = 21
    qkv = _r(T, Hq * D + Hkv * (D + Dv), dtype=dtype)
    qw, kw = 1 + 0.2 * _r(D, seed=1), 1 + 0.2 * _r(D, seed=2)
    pos = torch.arange(50, 50 + T, dtype=torch.int32).cuda()
    kp = torch.zeros(3, 128, Hkv, D, dtype=dtype, device="cuda")
    vp = torch.zeros(3, 128, Hkv, Dv, dtype=dtype, device="cuda")
    slots = (torch.randperm(384)[:T]).to(torch.int32).cuda()
    slots[3] = -1
    q = stream.qkv_prologue(qkv, heads, qw, kw, 1e-5, pos, (0.4, 16), slots, kp, vp)
    f = qkv.float()
    wq = O.rms_norm(f[:, :Hq * D].view(T, Hq, D), qw, 1e-5) * \
        O.query_temperature(pos.float(), 0.4, 16)[:, None, None]
    wk = O.rms_norm(f[:, Hq * D:(Hq + Hkv) * D].view(T, Hkv, D), kw, 1e-5)
    wv = qkv[:, (Hq + Hkv) * D:].view(T, Hkv, Dv)
    ok = slots >= 0
    _close(q, wq, dtype)
    _close(kp.view(-1, Hkv, D)[slots[ok].long()], wk[ok], dtype)
    assert torch.equal(vp.view(-1, Hkv, Dv)[slots[ok].long()], wv[ok])
    assert int((kp.view(384, -1).abs().sum(1) > 0).sum()) == T - 1


@pytest.mark.parametrize("V", [640, 1000, 77])
@pytest.mark.parametrize("dtype", DT)
def test_greedy_sampling_of_either_logit_type(V, dtype):
    from easydel_b200.ops import serving as S

    lg = _r(9, V, dtype=dtype)
    lg[2, 5] = lg[2, V - 1] = lg[2].max() + 1           # a tie: the first one wins
    tok, lp = S.sample(lg, want_logprob=True)
    assert tok.tolist() == lg.float().argmax(-1).tolist() and int(tok[2]) == 5
    want = torch.log_softmax(lg.float(), -1).gather(1, tok.long()[:, None])[:, 0]
    assert torch.allclose(lp, want, atol=1e-3)


# ------------------------------------------------------------------------------------------------ attention
def _paged(lens_kv, Hkv, D, Dv, dtype, seed=0):
    """Random keys / values of several sequences on shuffled pages; returns dense lists and the paged form."""
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // 128) for n in lens_kv]
    perm = (torch.randperm(sum(per), generator=g) + 1).tolist()
    table = torch.zeros(len(lens_kv), max(per), dtype=torch.int32)
    kp = torch.full((sum(per) + 1, 128, Hkv, D), 7.0, dtype=dtype)      # finite filler in unused places
    vp = torch.full((sum(per) + 1, 128, Hkv, Dv), -9.0, dtype=dtype)
    ks, vs = [], []
    for b, n in enumerate(lens_kv):
        pages = [perm.pop() for _ in range(per[b])]
        table[b, :per[b]] = torch.tensor(pages)
        k, v = torch.randn(n, Hkv, D, generator=g).to(dtype), torch.randn(n, Hkv, Dv, generator=g).to(dtype)
        k[3:4] *= 3
        for j in range(n):
            kp[pages[j // 128], j % 128], vp[pages[j // 128], j % 128] = k[j], v[j]
        ks.append(k)
        vs.append(v)
    return ks, vs, kp.cuda(), vp.cuda(), table.cuda()


def _expect(q, k, v, scale, sink):
    """The last len(q) positions of causal attention with a sink, in fp64."""
    n = q.shape[0]
    full = torch.cat([torch.zeros(k.shape[0] - n, *q.shape[1:]), q.float()])
    return O.sink_attention(full.double(), k.double(), v.double(), scale, sink.double())[-n:]


LAYOUTS = [(6, 6, 64, 88), (6, 2, 48, 24), (6, 1, 128, 72), (4, 4, 16, 128), (2, 1, 136, 144), (3, 3, 20, 12)]


@pytest.mark.parametrize("layout", LAYOUTS)
@pytest.mark.parametrize("dtype", DT)
def test_paged_attention_with_its_own_value_size(layout, dtype):
    from easydel_b200.ops import serving as S

    Hq, Hkv, D, Dv = layout
    kv, new = [300, 128, 1, 129, 700], [37, 128, 1, 2, 260]
    ks, vs, kp, vp, table = _paged(kv, Hkv, D, Dv, dtype)
    q = _r(sum(new), Hq, D, dtype=dtype)
    sink = _r(Hq, seed=5) + 1
    # one far key stands out for one late query of every long sequence: it must be found across pages
    at = 0
    for b, n in enumerate(new):
        if kv[b] > 200:
            k3 = ks[b][3].float()                            # three times as long as the other keys
            q[at + n - 1] = (k3 * (60 / 0.2 / k3.pow(2).sum(-1, keepdim=True))).repeat_interleave(Hq // Hkv, 0)
        at += n
    cu = _i32(*torch.tensor([0, *new]).cumsum(0).tolist())
    got = S.paged_attention(q, kp, vp, cu, _i32(*kv), table, max(new), scale=0.2, sinks=sink)
    want = torch.cat([_expect(c.cpu(), k, v, 0.2, sink.cpu()) for c, k, v in zip(torch.split(q, new), ks, vs)])
    _close(got.cpu(), want, dtype, 2)
    far = got[new[0] - 1].float().cpu()                    # that query returns (nearly) the far key's value
    assert (far - vs[0][3].float().repeat_interleave(Hq // Hkv, 0)).abs().max() < 0.1


@pytest.mark.parametrize("layout", LAYOUTS[:4])
@pytest.mark.parametrize("splits", [1, 3])
def test_decode_attention_with_its_own_value_size(layout, splits):
    from easydel_b200.ops import serving as S

    Hq, Hkv, D, Dv = layout
    kv = [1, 127, 128, 129, 640]
    ks, vs, kp, vp, table = _paged(kv, Hkv, D, Dv, torch.bfloat16, 1)
    q, sink = _r(5, Hq, D, dtype=torch.bfloat16), _r(Hq, seed=6) + 1
    assert S.decode_kernel_supports(q, kp, Dv)
    got = S.decode_attention(q, kp, vp, _i32(*kv), table, scale=0.3, sinks=sink, num_splits=splits)
    want = torch.cat([_expect(q[b:b + 1].cpu(), ks[b], vs[b], 0.3, sink.cpu()) for b in range(5)])
    _close(got.cpu(), want, torch.bfloat16, 2)


# ------------------------------------------------------------------------------------------------ HGRN2
@pytest.mark.parametrize("heads", [(5, 32, 56), (3, 48, 72), (2, 128, 128), (1, 200, 33), (2, 12, 10), (1, 300, 96)])
@pytest.mark.parametrize("dtype", DT)
def test_hgrn2_scan_and_decode(heads, dtype):
    """Several sequences of a step, states in shuffled slots, then single tokens; whole, segmented, and per step."""
    from easydel_b200.ops import ssm

    H, D, V = heads
    lens = [1, 17, 600, 2, 33]
    cu = _i32(*torch.tensor([0, *lens]).cumsum(0).tolist())
    T = sum(lens)
    proj = _r(T, 2 * H * D + H * V, dtype=dtype)
    bias, lower, norm = 2 + _r(H * D, seed=1), torch.rand(H * D).cuda(), 1 + 0.1 * _r(V, seed=2)
    slots = _i32(5, 0, 3, 1, 6)
    state = _r(7, H, D, V, seed=3)
    ref_state = state.cpu().clone()
    o = ssm.hgrn2_reference(proj.cpu(), heads, bias.cpu(), lower.cpu(), cu.cpu(), slots.cpu(), ref_state)
    want = O.rms_norm(o, norm.cpu(), 1e-6).reshape(T, H * V)
    for segments in (0, 3):
        st = state.clone()
        got = ssm.hgrn2(proj, heads, bias, lower, norm, 1e-6, cu, 600, slots, st, segments=segments)
        _close(got.cpu(), want, dtype, 4)
        _close(st.cpu(), ref_state, torch.float32, 4)
    one = _r(5, 2 * H * D + H * V, seed=9, dtype=dtype)
    cu1 = _i32(0, 1, 2, 3, 4, 5)
    o = ssm.hgrn2_reference(one.cpu(), heads, bias.cpu(), lower.cpu(), cu1.cpu(), slots.cpu(), ref_state)
    got = ssm.hgrn2(one, heads, bias, lower, norm, 1e-6, cu1, 1, slots, st)
    _close(got.cpu(), O.rms_norm(o, norm.cpu(), 1e-6).reshape(5, H * V), dtype, 4)
    _close(st.cpu(), ref_state, torch.float32, 4)
    assert torch.equal(st[2], state[2]) and torch.equal(st[4], state[4])       # other slots are untouched


# ------------------------------------------------------------------------------------------------ whole models
#: largest error of a row of logits, against their spread
LIMIT = {torch.float32: 3e-5, torch.bfloat16: 0.06}


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
@pytest.mark.parametrize("dtype", DT)
def test_model_whole_portions_and_decoding(tmp_path, name, dtype):
    cfg, w, model = C.make(tmp_path, name, dtype, "cuda")
    toks = C.tokens(270, cfg["vocab"], 4)
    want = O.forward(cfg, w, toks)
    got = model(input_ids=torch.tensor([toks], device="cuda")).logits[0].cpu()
    assert got.dtype == torch.float32 and C.error(got, want) < LIMIT[dtype]
    rep = C.replayer(model)
    for i, cuts in enumerate([[270], [200, 1], [2], [127, 1, 1, 1, 100, 3]]):
        assert C.error(C.run_cut(rep, f"r{i}", toks, cuts), want) < LIMIT[dtype], cuts
    assert rep.engine.runner.use_graphs and rep.engine.runner._graphs      # single tokens replayed a captured step


@pytest.mark.parametrize("mutate", ["no_shift", "no_sink", "no_q_temp", "kv_head", "no_loop_step"])
def test_a_wrong_mechanism_would_show(tmp_path, mutate):
    cfg, w, model = C.make(tmp_path, "looped", torch.bfloat16, "cuda")
    toks = C.tokens(60, cfg["vocab"])
    got = model(input_ids=torch.tensor([toks], device="cuda")).logits[0].cpu()
    assert C.error(got, O.forward(cfg, w, toks, mutate=mutate)) > 2 * LIMIT[torch.bfloat16]


@pytest.mark.parametrize("dtype", DT)
def test_mixed_batches_against_each_request_alone(tmp_path, dtype):
    """Portions beside single tokens, requests that pause, pages and slots taken over from requests that ended."""
    import random

    cfg, w, model = C.make(tmp_path, "looped", dtype, "cuda")
    rep = C.replayer(model, max_tokens=1024)
    rnd = random.Random(5)
    lens = [300, 1, 64, 129, 257, 2, 130, 40]
    seqs = {f"s{i}": C.tokens(n, cfg["vocab"], i) for i, n in enumerate(lens)}
    at, got, waiting, live = dict.fromkeys(seqs, 0), {n: [] for n in seqs}, list(seqs), []
    while waiting or live:
        while waiting and len(live) < 4:
            live.append(waiting.pop(0))
        entries, end, members = [], [], []
        for n in rnd.sample(live, rnd.randint(1, len(live))):
            k = min(rnd.choice([1, 1, 1, 2, 29, 128]), len(seqs[n]) - at[n])
            entries.append({"id": n, "tokens": seqs[n][at[n]:at[n] + k], "want": list(range(k))})
            members.append((n, k))
            at[n] += k
            if at[n] == len(seqs[n]):
                end.append(n)
        lg = rep.step(entries, end)
        for n, k in members:
            got[n].append(lg[:k])
            lg = lg[k:]
        live = [n for n in live if n not in end]
    for n, toks in seqs.items():
        assert C.error(torch.cat(got[n]), O.forward(cfg, w, toks)) < LIMIT[dtype], n


def test_greedy_generation_and_long_decoding(tmp_path):
    """The engine's own scheduler, asynchronous and through captured decode steps, in 32 bits against the oracle; long
    enough that decoding crosses a page."""
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cuda")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (3, 120, 70)]
    eng = eSurge(model, max_model_len=512, max_num_seqs=2, num_pages=8, max_num_batched_tokens=64)
    outs = eng.generate(prompts, SamplingParams(max_tokens=24, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        toks = p + o.outputs[0].token_ids
        lg = O.forward(cfg, w, toks)[len(p) - 1:-1]
        top = lg.topk(2).values
        pick = lg.argmax(-1).tolist()
        for i, t in enumerate(o.outputs[0].token_ids):       # equal wherever the oracle's choice is not a tie
            assert t == pick[i] or float(top[i, 0] - top[i, 1]) < 1e-4, (i, t, pick[i])
    assert eng.runner.timings["graph_steps"] > 0
    out = eng.generate([prompts[0]], SamplingParams(max_tokens=260, temperature=0.0, ignore_eos=True))[0]
    toks = prompts[0] + out.outputs[0].token_ids
    pick = O.forward(cfg, w, toks)[len(prompts[0]) - 1:-1].argmax(-1).tolist()
    assert sum(a != b for a, b in zip(out.outputs[0].token_ids, pick)) <= 1
    sampled = eng.generate([prompts[0]], SamplingParams(max_tokens=8, temperature=0.9, top_k=20, seed=3))[0]
    assert len(sampled.outputs[0].token_ids) <= 8
    eng.close()


def test_generate_with_padding(tmp_path):
    cfg, w, model = C.make(tmp_path, "looped", torch.float32, "cuda")
    a, b = C.tokens(9, cfg["vocab"], 1), C.tokens(5, cfg["vocab"], 2)
    ids = torch.tensor([a, [0] * 4 + b]).cuda()
    mask = torch.tensor([[1] * 9, [0] * 4 + [1] * 5]).cuda()
    seqs = model.generate(ids, attention_mask=mask, max_new_tokens=6).sequences.cpu()
    for row, p in ((seqs[0], a), (seqs[1], b)):
        new = row[-6:].tolist()
        assert O.forward(cfg, w, p + new)[len(p) - 1:-1].argmax(-1).tolist() == new
