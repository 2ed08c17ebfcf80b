"""Ninisun on the GPU: every kernel of the family against plain forms, whole models against a plain restatement."""

import math
import types

import ninisun_cases as C
import oracle_ninisun as O
import pytest
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


def _status():
    from easydel_b200.ops import _lib

    _lib.check_status(torch.device("cuda", 0))


# ------------------------------------------------------------------------------------------------ kernels of the stream
@pytest.mark.parametrize("W", [60, 77, 352, 3000, 8192, 9000])
@pytest.mark.parametrize("dtype", DT)
def test_normed_branch_joins_the_stream(W, dtype):
    from easydel_b200.ops import stream

    x, y = 3 * _r(37, W), 0.2 * _r(37, W, seed=1)
    wb, ls, w = 1 + 0.3 * _r(W, seed=2), _r(W, seed=3), 1 + 0.3 * _r(W, seed=4)
    for scale in (ls, None):
        s, h = stream.add_norm(x.clone(), stream.NormedBranch(y, wb, 1e-3, scale), 1.0, w, 1e-5, dtype)
        b = O.rms_norm(y.double(), wb.double(), 1e-3)
        want = x.double() + (b if scale is None else b * scale.double())
        _close(s, want, torch.float32)
        _close(h, O.rms_norm(want, w.double(), 1e-5), dtype)


@pytest.mark.parametrize("act,f", [("gelu_tanh", O.gelu_tanh), ("silu", lambda z: z * O.sigmoid(z))])
@pytest.mark.parametrize("T,F", [(5, 11), (64, 1000), (3, 12)])
@pytest.mark.parametrize("dtype", DT)
def test_gated_unit(act, f, T, F, dtype):
    from easydel_b200.ops import stream

    gu = 3 * _r(T, 2 * F, seed=2, dtype=dtype)
    want = f(gu[:, :F].double()) * gu[:, F:].double()
    _close(stream.gated_unit(gu, act), want, dtype)


POSITIONS = torch.tensor([*range(11), *range(1000, 1005), 30001, 99999, 100000, 100001, 250000], dtype=torch.int32)


@pytest.mark.parametrize("heads,dims", [((4, 2, 48, 24), 32), ((3, 1, 20, 12), 6), ((16, 2, 128, 64), 128), ((2, 2, 7, 3), 2),
                                        ((12, 4, 64, 128), 0), ((2, 1, 24, 8), 8), ((32, 8, 128, 64), 32),
                                        ((64, 8, 128, 128), 16), ((96, 8, 128, 16), 8), ((5, 5, 9, 8), 8)])
@pytest.mark.parametrize("bias", [False, True])
@pytest.mark.parametrize("blend", [False, True])
@pytest.mark.parametrize("dtype", DT)
def test_attention_prologue(heads, dims, bias, blend, dtype):
    """Biases, rotated neighbours with a magnitude, blended values, keys and values on their pages."""
    from easydel_b200.ops import rotation, stream

    H, G, D, V = heads
    T = 21
    ld = H * D + G * (D + V)
    qkv = _r(T, ld + (8 if dims else 3), dtype=dtype)[:, :ld]
    b = _r(ld, seed=1) if bias else None
    first = _r(T, G * V + 16, seed=2, dtype=dtype)[:, :G * V].unflatten(1, (G, V)) if blend else None
    lam = torch.tensor(0.3, device="cuda") if blend else None
    rot = {"base": 700.0, "dims": dims, "scaling": {"factor": 3.0, "original": 500, "fast": 8.0, "slow": 1.0}}
    freq = rotation.pair_frequencies(700.0, dims, "cuda", rot["scaling"]) if dims else None
    kp = torch.zeros(3, 128, G, D, dtype=dtype, device="cuda")
    vp = torch.zeros(3, 128, G, V, dtype=dtype, device="cuda")
    slots = torch.randperm(384, generator=torch.Generator().manual_seed(2))[:T].to(torch.int32).cuda()
    slots[3] = -1
    args = ("neighbours", rotation.magnitude(rot["scaling"]), b)
    q = stream.qkv_rotary_prologue(qkv, heads, None, None, 0.0, POSITIONS.cuda(), freq, slots, kp, vp, *args, first, lam)
    _status()
    f = qkv.cpu().double() + (b.cpu().double() if bias else 0.0)
    turn = (lambda x: O.rotate(x, POSITIONS, rot)) if dims else (lambda x: x)
    want_q = turn(f[:, :H * D].reshape(T, H, D))
    want_k = turn(f[:, H * D:(H + G) * D].reshape(T, G, D))
    want_v = f[:, (H + G) * D:]
    if blend:
        want_v = (1 - lam.cpu().double()) * want_v + lam.cpu().double() * first.cpu().double().flatten(1)
    _close(q.cpu(), want_q, dtype)
    ok = (slots >= 0).cpu()
    at = slots.cpu()[ok].long()
    _close(kp.view(384, G, D).cpu()[at], want_k[ok], dtype)
    _close(vp.view(384, -1).cpu()[at], want_v[ok], dtype)
    assert int((kp.view(384, -1).abs().sum(1) > 0).sum()) == T - 1
    # many tokens (a block walks several), the same rows over and over
    n = 90
    kp2, vp2 = (torch.zeros(T * n // 128 + 1, *p.shape[1:], dtype=dtype, device="cuda") for p in (kp, vp))
    many = stream.qkv_rotary_prologue(qkv.repeat(n, 1), heads, None, None, 0.0, POSITIONS.cuda().repeat(n), freq,
                                      torch.arange(T * n, dtype=torch.int32, device="cuda"), kp2, vp2, *args,
                                      first.repeat(n, 1, 1) if blend else None, lam)
    many, k, v = many.view(n, T, H, D), kp2.view(-1, G, D)[:T * n].view(n, T, G, D), vp2.view(-1, G * V)[:T * n].view(n, T, -1)
    assert torch.equal(many, many[:1].expand_as(many)) and torch.equal(k, k[:1].expand_as(k)) and torch.equal(v, v[:1].expand_as(v))
    _close(many[0].cpu(), want_q, dtype)
    _close(k[0].cpu(), want_k, dtype)
    _close(v[0].cpu(), want_v, dtype)


def test_halves_take_biases_magnitudes_and_blends_too():
    from easydel_b200.ops import rotation, stream

    for heads, dims in (((6, 2, 64, 32), 32), ((3, 1, 10, 4), 6)):
        H, G, D, V = heads
        T, ld = 21, H * D + G * (D + V)
        qkv, b, first, lam = _r(T, ld), _r(ld, seed=1), _r(T, G, V, seed=2), torch.tensor(0.7, device="cuda")
        freq = rotation.pair_frequencies(700.0, dims, "cuda")
        kp, vp = torch.zeros(1, 128, G, D, device="cuda"), torch.zeros(1, 128, G, V, device="cuda")
        slots = torch.arange(T, dtype=torch.int32, device="cuda")
        args = (heads, None, None, 0.0, POSITIONS.cuda(), freq)
        q = stream.qkv_rotary_prologue(qkv, *args, slots, kp, vp, "halves", 1.25, b, first, lam)
        want = stream.rotary_rows(qkv, *args, "halves", 1.25, b, first, lam)
        for g, w in zip((q, kp[0, :T], vp[0, :T]), want):
            _close(g, w, torch.float32)
    _status()


# ------------------------------------------------------------------------------------------------ attention
def _layer(scale, window, keep):
    return types.SimpleNamespace(scale=scale, sliding_window=window, keep_first=keep, softcap=0.0, sinks=None)


def _step(shape, layer, lens, new, dtype, spike=(), seed=0, bias=None):
    """Keys and values of sequences of ``lens`` keys on shuffled pages, queries of their last ``new`` tokens, and what
    attention has to give. ``spike``: key positions (counted back from the sequence's last query) made to stand out;
    ``bias``: sigmoid weights."""
    from easydel_b200.caching.paged import PagedBatchMeta, PagedLayerView

    H, G, D, V = shape
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // 128) for n in lens]
    perm = (torch.randperm(sum(per), generator=g) + 1).tolist()
    table = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    kp = torch.full((sum(per) + 1, 128, G, D), 5.0, dtype=dtype)                 # finite filler in unused places
    vp = torch.full((sum(per) + 1, 128, G, V), 5.0, dtype=dtype)
    q = torch.randn(sum(new), H, D, generator=g).to(dtype)
    want, at = [], 0
    for b, (n, m) in enumerate(zip(lens, new)):
        ids = [perm.pop() for _ in range(per[b])]
        table[b, :per[b]] = torch.tensor(ids)
        k, v = torch.randn(n, G, D, generator=g).to(dtype), torch.randn(n, G, V, generator=g).to(dtype)
        for back in spike:
            if 0 <= n - 1 - back:
                k[n - 1 - back] *= 4
                v[n - 1 - back] *= 4
        if layer.keep_first and n > layer.keep_first:        # the last kept key and the first one that is not
            v[layer.keep_first - 1:layer.keep_first + 1] *= 6
        for j in range(0, n, 128):
            c = min(128, n - j)
            kp[ids[j // 128], :c], vp[ids[j // 128], :c] = k[j:j + c], v[j:j + c]
        if layer.sliding_window:                             # pages that no query of the step can see are given back
            first = max(0, n - m - layer.sliding_window + 1) // 128
            table[b, -(-layer.keep_first // 128):first] = 0
        full = torch.cat([torch.zeros(n - m, H, D, dtype=torch.double), q[at:at + m].double()])
        args = (full, k.double(), v.double(), layer.scale)
        mask = (layer.sliding_window, layer.keep_first)
        o = O.softmax_heads(*args, *mask) if bias is None else O.sigmoid_heads(*args, bias.cpu().double(), *mask)
        want.append(o[-m:])
        at += m
    cu = torch.tensor([0, *new]).cumsum(0).to(torch.int32).cuda()
    meta = PagedBatchMeta(cu_q=cu, kv_lens=_i32(*lens), page_table=table.cuda(), slot_mapping=None, max_q=max(new),
                          num_seqs=len(lens), spans=list(zip(new, lens)))
    return q.cuda(), PagedLayerView(kp.cuda(), vp.cuda()), meta, torch.cat(want).cuda()


SHAPES = [(6, 2, 48, 24), (16, 2, 128, 64), (34, 2, 64, 128), (3, 1, 20, 12), (4, 4, 16, 40), (1, 1, 8, 8), (6, 2, 96, 96),
          (4, 1, 136, 72)]
MASKS = [(None, 0), (1, 1), (44, 5), (128, 32), (60, 130), (300, 129), (20, 260)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("sigmoid", [False, True])
@pytest.mark.parametrize("dtype", DT)
def test_attention_decode(shape, window, keep, sigmoid, dtype):
    _attention(shape, window, keep, sigmoid, dtype, [1, 31, 44, 45, 49, 128, 129, 300, 301, 517], None)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,keep", MASKS)
@pytest.mark.parametrize("sigmoid", [False, True])
@pytest.mark.parametrize("dtype", DT)
def test_attention_portions_beside_single_tokens(shape, window, keep, sigmoid, dtype):
    _attention(shape, window, keep, sigmoid, dtype, [5, 290, 700, 130, 400, 129, 760, 64], [1, 1, 2, 130, 257, 3, 300, 64])


def _attention(shape, window, keep, sigmoid, dtype, lens, new):
    from easydel_b200.ops.serving import SigmoidWeights

    H, V = shape[0], shape[3]
    layer = _layer(shape[2] ** -0.5, window, keep)
    edge = (window or 1) - 1
    bias = 1.5 * _r(H, seed=5) - 2.0 if sigmoid else None
    q, view, meta, want = _step(shape, layer, lens, new or [1] * len(lens), dtype, spike=(edge, edge + 1, 127, 128), bias=bias)
    T = q.shape[0]
    for splits in (1, 3) if new is None else (1,):
        meta.num_splits = splits
        got = view.attend_pages(layer, q, meta)
        _status()
        if not sigmoid:
            _close(got, want, dtype, 2.5)
            continue
        # weights that stand alone, with and without gate and factor, into columns of a wider row
        gate = _r(T, H + 5, seed=6, dtype=dtype)[:, :H]
        out = torch.full((T, H * V + 24), 7.0, dtype=dtype, device="cuda")
        got = view.attend_pages(layer, q, meta, sigmoid=SigmoidWeights(bias, gate, 1.7),
                                out=out[:, 8:8 + H * V].unflatten(1, (H, V)))
        _status()
        assert got.data_ptr() == out.data_ptr() + 8 * out.element_size()
        _close(got, want * 1.7 * O.sigmoid(gate.double())[..., None], dtype, 2.5)
        assert bool((out[:, :8] == 7).all()) and bool((out[:, 8 + H * V:] == 7).all())
        out = torch.empty(T, H * V + 3, dtype=dtype, device="cuda")[:, 1:1 + H * V].unflatten(1, (H, V))      # no alignment
        _close(view.attend_pages(layer, q, meta, sigmoid=SigmoidWeights(bias), out=out), want, dtype, 2.5)
        _close(out, want, dtype, 2.5)
        _status()


@pytest.mark.parametrize("dtype", DT)
@pytest.mark.parametrize("bias", [-30.0, -8.0, 0.0, 20.0])
def test_sigmoid_weights_of_every_size(bias, dtype):
    """Thousands of tiny weights add up to something, saturated ones to the plain sum of the values."""
    from easydel_b200.ops.serving import SigmoidWeights

    shape = (4, 2, 64, 64)
    layer = _layer(0.3, None, 0)
    b = torch.full((4,), bias, device="cuda")
    for new in ([1, 1], [3, 200]):
        q, view, meta, want = _step(shape, layer, [2000, 700], new, dtype, bias=b)
        _close(view.attend_pages(layer, q, meta, sigmoid=SigmoidWeights(b)), want, dtype, 2.5)
    _status()


def test_window_edges_and_kept_tokens_are_seen_and_not_seen():
    """One key stands far above the rest: a query that sees it copies its value, the others do not."""
    from easydel_b200.caching.paged import PagedLayerView

    n, H, G, D = 520, 4, 2, 64
    for dtype in DT:
        for window, keep in ((16, 2), (128, 128), (200, 1), (40, 129)):
            layer = _layer(1.0, window, keep)
            q, view, meta, _ = _step((H, G, D, D), layer, [n], [n], dtype)
            ids = meta.page_table[0, :5].long()
            q = torch.zeros_like(q)
            q[..., 0] = 8.0
            for key in (0, 1, 2, 127, 128, 129, 190):
                kp = torch.zeros_like(view.k_pages)
                kp[ids[key // 128], key % 128, :, 0] = 8.0        # a score of 64; the others have 0
                got = PagedLayerView(kp, view.v_pages).attend_pages(layer, q, meta)
                value = view.v_pages[ids[key // 128], key % 128].double().repeat_interleave(H // G, 0)
                err = ((got.double() - value).abs().amax((1, 2)) / value.abs().max()).tolist()
                for i in range(n):
                    seen = 0 <= i - key and (i - key < window or key < keep)
                    assert (err[i] < 0.02) == seen, (dtype, window, keep, key, i, err[i])
    _status()


# ------------------------------------------------------------------------------------------------ generalised delta rule
def _delta_case(H, D, V, rank, T, dtype, pad=3, seed=0):
    from easydel_b200.ops import ssm

    widths = (H * D, H * D, H * V, H * D, H * V, rank)
    rows = _r(T, sum(widths) + pad, seed=seed, dtype=dtype)
    cols = ssm.DeltaColumns(*torch.split(rows[:, :sum(widths)], widths, -1))
    wt = ssm.DeltaWeights(_r(H * D, rank, seed=1, dtype=dtype), 1.5 * _r(H * D, seed=2) - 3, _r(H * D, seed=3),
                          1 + 0.2 * _r(H * V, seed=4), math.exp(-0.5), 1e-6, 1e-5)
    return cols, wt


def _delta_oracle(cols, wt, H, S, scale):
    T = cols.r.shape[0]
    h3 = lambda t: t.double().reshape(T, H, -1)  # noqa: E731
    z = torch.tanh(cols.x.double()) @ wt.w2.double().t() + wt.w0.double()
    w, a = torch.exp(-wt.rate * O.sigmoid(z)), O.sigmoid(cols.a.double() + wt.a0.double())
    o, S = O.delta_rule(h3(cols.r), h3(w), h3(cols.k), h3(a), h3(cols.v), S)
    o = (o / torch.sqrt((o * o).mean(-1, keepdim=True) + wt.eps)).reshape(T, -1)
    return o * wt.norm.double() * O.sigmoid(cols.g.double()) * scale, S


DELTA_SIZES = [(3, 16, 16, 8), (2, 32, 32, 16), (5, 7, 7, 5), (4, 64, 64, 64), (2, 128, 128, 24), (1, 100, 36, 12),
               (1, 192, 192, 16), (1, 512, 40, 4), (2, 20, 130, 33)]


@pytest.mark.parametrize("H,D,V,rank", DELTA_SIZES)
@pytest.mark.parametrize("dtype", DT)
def test_generalised_delta_rule(H, D, V, rank, dtype):
    """Unequal sequences in one step, each from the state of its own slot; then single tokens from the states it left."""
    from easydel_b200.ops import ssm

    lens = [1, 70, 2, 17, 8, 9]
    T, slots = sum(lens), [5, 0, 3, 6, 1, 2]
    cols, wt = _delta_case(H, D, V, rank, T, dtype)
    cu = torch.tensor([0, *lens]).cumsum(0).to(torch.int32).cuda()
    state = 0.3 * _r(8, H, D, V, seed=7)
    old = state.clone()
    out = torch.full((T, H * V + 16), 7.0, dtype=dtype, device="cuda")
    got = ssm.generalized_delta_rule(cols, (H, D, V), wt, cu, max(lens), _i32(*slots), state, 0.8, out[:, 8:8 + H * V])
    assert bool((out[:, :8] == 7).all()) and bool((out[:, 8 + H * V:] == 7).all())
    at = 0
    slack = 4 if dtype == torch.float32 else 2      # the rows pass rounds tanh(x) to the operand type: decays follow
    for n, s in zip(lens, slots):
        part = ssm.DeltaColumns(*(t[at:at + n] for t in vars(cols).values()))
        want, S = _delta_oracle(part, wt, H, old[s].double(), 0.8)
        _close(got[at:at + n], want, dtype, slack)
        _close(state[s], S, torch.float32 if dtype == torch.float32 else torch.bfloat16, 3)
        at += n
    for s in (4, 7):
        assert torch.equal(state[s], old[s])
    # one token each
    cols, wt = _delta_case(H, D, V, rank, 3, dtype, seed=11)
    rows = _i32(2, 7, 0)
    before = state.clone()
    got = ssm.generalized_delta_rule(cols, (H, D, V), wt, _i32(0, 1, 2, 3), 1, rows, state, 0.8)
    for b, s in enumerate(rows.tolist()):
        part = ssm.DeltaColumns(*(t[b:b + 1] for t in vars(cols).values()))
        want, S = _delta_oracle(part, wt, H, before[s].double(), 0.8)
        _close(got[b:b + 1], want, dtype, 4 if dtype == torch.float32 else 1)
        _close(state[s], S, torch.float32, 2)          # the decode form keeps tanh(x) in 32 bits
    assert all(torch.equal(state[s], before[s]) for s in range(8) if s not in rows.tolist())


@pytest.mark.parametrize("dtype", DT)
def test_delta_rule_over_a_long_sequence(dtype):
    """Thousands of tokens: what 32-bit arithmetic alone does to the state stays small; cuts do not matter."""
    from easydel_b200.ops import ssm

    H, D, rank, T = 2, 64, 16, 3000
    cols, wt = _delta_case(H, D, D, rank, T, dtype)
    state = torch.zeros(2, H, D, D, device="cuda")
    got = ssm.generalized_delta_rule(cols, (H, D, D), wt, _i32(0, T), T, _i32(1), state)
    want, S = _delta_oracle(cols, wt, H, None, 1.0)
    _close(got, want, dtype, 10 if dtype == torch.float32 else 3)
    if dtype == torch.float32:
        _close(state[1], S, dtype, 10)
    parts, st, at = [], torch.zeros(2, H, D, D, device="cuda"), 0
    for n in (2, 1, 129, 1000, 3, T - 1135):
        part = ssm.DeltaColumns(*(t[at:at + n] for t in vars(cols).values()))
        parts.append(ssm.generalized_delta_rule(part, (H, D, D), wt, _i32(0, n), n, _i32(0), st))
        at += n
    _close(torch.cat(parts), got, dtype, 10 if dtype == torch.float32 else 3)


# ------------------------------------------------------------------------------------------------ whole models
def _check(cfg, w, got, toks, dtype):
    floor = 3e-5 if dtype == torch.float32 else 1.5 * C.bf16_floor(cfg, w, toks)
    err = C.error(got, O.forward(cfg, w, toks))
    assert err < floor, (err, floor)


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
@pytest.mark.parametrize("cuts", [[400], [370, 1], [2, 3, 1, 129, 64]])
@pytest.mark.parametrize("dtype", DT)
def test_models_in_portions_and_decoding(tmp_path, name, cuts, dtype):
    cfg, w, model = C.make(tmp_path, name, dtype, "cuda")
    toks = C.tokens(400, cfg["vocab"], 3)
    rep = C.replayer(model)
    assert rep.engine.runner.use_graphs
    _check(cfg, w, C.run_cut(rep, "a", toks, cuts), toks, dtype)


@pytest.mark.parametrize("dtype", DT)
def test_far_keys_under_sigmoid_weights(tmp_path, dtype):
    """A twin layer alone finds one token far back, in a prompt and in decoding."""
    cfg = O.random_config([O.parallel((4, 2, 64, 64, 0.4, 16, 1e6, C.YARN), (2, 16), (1.0, 0.1))], 64, 96)
    w = O.random_weights(cfg, 1)
    w["l0.mix.left.q"] = (w["l0.mix.left.q"].float() * 2).to(torch.bfloat16)
    w["l0.mix.left.pb"] = (w["l0.mix.left.pb"].float() - 3).to(torch.bfloat16)
    cfg, w, model = C.make(tmp_path, "far", dtype, "cuda", cfg=cfg, weights=w)
    toks = C.tokens(420, 96, 3)
    assert C.error(O.forward(cfg, w, toks, mutate="softmax"), O.forward(cfg, w, toks)) > 0.1
    for cuts in ([420], [300, 1], [129, 2, 64]):
        _check(cfg, w, C.run_cut(C.replayer(model), "a", toks, cuts), toks, dtype)


@pytest.mark.parametrize("name", ["mixed", "wide"])
@pytest.mark.parametrize("dtype", DT)
def test_mixed_batches_reuse_pages_and_slots(tmp_path, name, dtype):
    cfg, w, model = C.make(tmp_path, name, dtype, "cuda")
    rep = C.replayer(model, max_tokens=768, max_requests=3)
    pool_free = [m.pool.num_free for m in rep.engine.kv.managers]
    seqs = {n: C.tokens(k, cfg["vocab"], i) for i, (n, k) in enumerate(
        [("a", 300), ("b", 5), ("c", 90), ("d", 259), ("e", 2)])}
    plan = [[("a", 200), ("b", 1)], [("a", 98), ("b", 2), ("c", 64)], [("b", 2), ("a", 1)], [("a", 1), ("c", 1), ("d", 230)],
            [("d", 2), ("c", 25), ("e", 1)], [("d", 26), ("e", 1)], [("d", 1)]]
    for n, lg in C.feed(rep, plan, seqs).items():
        if len(seqs[n]) > 50 or dtype == torch.float32:
            _check(cfg, w, lg, seqs[n], dtype)
    assert [m.pool.num_free for m in rep.engine.kv.managers] == pool_free


@pytest.mark.parametrize("dtype", DT)
def test_cuts_and_company_do_not_matter(tmp_path, dtype):
    """The same tokens whole, in portions and beside other requests: equal beyond rounding."""
    cfg, w, model = C.make(tmp_path, "mixed", dtype, "cuda")
    toks = C.tokens(300, cfg["vocab"], 5)
    whole = C.run_cut(C.replayer(model), "a", toks, [300])
    rep = C.replayer(model)
    rep.step([{"id": "x", "tokens": C.tokens(77, cfg["vocab"], 9), "want": []}])
    parts, at = [], 0
    for i, n in enumerate([2, 127, 1, 1, 64, 3, 101, 1]):
        lg = rep.step([{"id": "x", "tokens": [i], "want": []}, {"id": "a", "tokens": toks[at:at + n], "want": range(n)}])
        parts.append(lg)
        at += n
    floor = 1e-5 if dtype == torch.float32 else 1.5 * C.bf16_floor(cfg, w, toks)
    assert at == 300 and C.error(torch.cat(parts), whole) < floor


def test_greedy_generation_through_the_engine(tmp_path):
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    cfg, w, model = C.make(tmp_path, "mixed", torch.float32, "cuda")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (1, 13, 200, 40)]
    eng = eSurge(model, max_model_len=256, max_num_seqs=3, num_pages=6, max_num_batched_tokens=48)
    outs = eng.generate(prompts, SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == C.greedy(cfg, w, p, 8)
    assert eng.runner.timings["graph_steps"] > 0
    _status()


def test_long_16_bit_generation(tmp_path):
    from easydel_b200.inference import SamplingParams
    from easydel_b200.inference.esurge import eSurge

    cfg, w, model = C.make(tmp_path, "wide", torch.bfloat16, "cuda")
    eng = eSurge(model, max_model_len=1024, max_num_seqs=4, num_pages=32)
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (5, 300, 64)]
    sp = SamplingParams(max_tokens=400, temperature=0.0, ignore_eos=True)
    first = [o.outputs[0].token_ids for o in eng.generate(prompts, sp)]
    assert [len(t) for t in first] == [400] * 3
    # every generated token is (nearly) the best one of the plain form given the tokens before it
    for p, t in zip(prompts, first):
        lg = O.forward(cfg, w, p + t)[len(p) - 1:-1]
        gap = (lg.max(-1).values - lg.gather(1, torch.tensor(t)[:, None])[:, 0]) / lg.std()
        assert float(gap.quantile(0.95)) < 0.3
    _status()
