"""Gasetar on the GPU: every kernel of the family against plain forms, whole models against a plain restatement."""

import types

import gasetar_cases as C
import oracle_gasetar as O
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
@pytest.mark.parametrize("W", [60, 77, 352, 3000, 9000])
@pytest.mark.parametrize("dtype", DT)
def test_sum_of_the_branches_and_norm(W, dtype):
    from easydel_b200.ops import stream
    from easydel_b200.ops.moe_kernels import ExpertRows

    x, y, w = 3 * _r(37, W), _r(37, W, seed=1), 1 + 0.3 * _r(W, seed=2)
    s, h = stream.add_norm(x.clone(), y, 0.7, w, 1e-5, dtype)
    want = x.double() + 0.7 * y.double()
    _close(s, want, torch.float32)
    _close(h, O.rms_norm(want, w.double(), 1e-5), dtype)
    # expert rows (some of them nobody's) beside fp32 rows of the same branch
    ys, wts = _r(200, W, seed=3, dtype=dtype), torch.rand(37, 6).cuda()
    pos = torch.randint(0, 200, (37, 6), generator=torch.Generator().manual_seed(4)).to(torch.int32).cuda()
    pos[5, 1] = -1
    rows = (ys.double()[pos.clamp_min(0).long()] * (wts * (pos >= 0)).double()[..., None]).sum(1)
    for base in (None, y):
        s, h = stream.add_norm(x.clone(), ExpertRows(ys, wts, pos.reshape(-1).contiguous(), base), 1.3, w, 1e-5, dtype)
        want = x.double() + 1.3 * (rows if base is None else rows + base.double())
        _close(s, want, torch.float32)
        _close(h, O.rms_norm(want, w.double(), 1e-5), dtype)
    s, h = stream.add_norm(x, None, 1.3, w, 1e-5, dtype)
    assert s is x
    _close(h, O.rms_norm(x.double(), w.double(), 1e-5), dtype)


@pytest.mark.parametrize("n", [(5, 77), (64, 1000), (1, 3)])
def test_capped_logits_gated_unit_and_scaled_embedding(n):
    from easydel_b200.ops import stream

    z = 20 * _r(*n)
    for scale, cap in ((0.3, 5.0), (1.0, 30.0), (2.5, 0.0)):
        _close(stream.scale_cap(z.clone(), scale, cap), O.soft_cap(scale * z.double(), cap), torch.float32)
    for dtype in DT:
        table = _r(50, n[1], seed=1, dtype=dtype)
        ids = torch.tensor([0, 49, 7], device="cuda")
        right = torch.empty(3, n[1], dtype=dtype, device="cuda")
        x = stream.embed(table, ids, right, 13.7)
        _close(x, table[ids].double() * 13.7, torch.float32)
        _close(right, table[ids].double() * 13.7, dtype)
        for F in (24, 11):
            gu = 3 * _r(n[0], 2 * F, seed=2, dtype=dtype)
            _close(stream.gated_unit(gu), O.silu(gu[:, :F].double()) * gu[:, F:].double(), dtype)
    _status()


POSITIONS = torch.tensor([*range(11), *range(1000, 1005), 30001, 99999, 100000, 100001, 250000], dtype=torch.int32)


@pytest.mark.parametrize("heads,dims", [((4, 2, 48, 24), 32), ((3, 1, 20, 12), 6), ((16, 2, 128, 64), 128), ((2, 2, 7, 3), 2),
                                        ((12, 4, 64, 128), 0), ((2, 1, 24, 8), 8), ((32, 8, 128, 64), 32),
                                        ((64, 8, 128, 128), 16), ((96, 8, 128, 16), 0)])
@pytest.mark.parametrize("dtype", DT)
def test_attention_prologue(heads, dims, dtype):
    """Full-width norms, rotated halves, keys and values on their pages; at positions far beyond any table too."""
    from easydel_b200.ops import rotation, stream

    H, G, D, V = heads
    T = 21
    ld = H * D + G * (D + V)
    qkv = _r(T, ld + (8 if dims else 3), dtype=dtype)[:, :ld]
    qw, kw = 1 + 0.3 * _r(H * D, seed=1), 1 + 0.3 * _r(G * D, seed=2)
    rot = {"base": 700.0, "dims": dims, "scaling": dict(factor=3.0, low=1.0, high=4.0, original=500)}
    freq = rotation.pair_frequencies(700.0, dims, "cuda", rot["scaling"]) if dims else None
    kp = torch.zeros(3, 128, G, D, dtype=dtype, device="cuda")
    vp = torch.zeros(3, 128, G, V, dtype=dtype, device="cuda")
    slots = torch.randperm(384, generator=torch.Generator().manual_seed(2))[:T].to(torch.int32).cuda()
    slots[3] = -1
    q = stream.qkv_rotary_prologue(qkv, heads, qw, kw, 1e-4, POSITIONS.cuda(), freq, slots, kp, vp)
    _status()
    f = qkv.cpu().double()
    turn = (lambda x: O.rotate_half(x, POSITIONS, rot)) if dims else (lambda x: x)
    want_q = turn(O.rms_norm(f[:, :H * D], qw.cpu().double(), 1e-4).view(T, H, D))
    want_k = turn(O.rms_norm(f[:, H * D:(H + G) * D], kw.cpu().double(), 1e-4).view(T, G, D))
    _close(q.cpu(), want_q, dtype)
    ok = (slots >= 0).cpu()
    at = slots.cpu()[ok].long()
    _close(kp.view(384, G, D).cpu()[at], want_k[ok], dtype)
    assert torch.equal(vp.view(384, -1).cpu()[at], qkv.cpu()[ok][:, (H + G) * D:])
    assert int((kp.view(384, -1).abs().sum(1) > 0).sum()) == T - 1
    # many tokens (a block walks several), the same rows over and over
    n = 90
    kp2, vp2 = (torch.zeros(T * n // 128 + 1, *p.shape[1:], dtype=dtype, device="cuda") for p in (kp, vp))
    many = stream.qkv_rotary_prologue(qkv.repeat(n, 1), heads, qw, kw, 1e-4, POSITIONS.cuda().repeat(n), freq,
                                      torch.arange(T * n, dtype=torch.int32, device="cuda"), kp2, vp2)
    many, k = many.view(n, T, H, D), kp2.view(-1, G, D)[:T * n].view(n, T, G, D)
    assert torch.equal(many, many[:1].expand_as(many)) and torch.equal(k, k[:1].expand_as(k))
    _close(many[0], q, dtype)          # rows of another pitch may take another form of the kernel
    _close(k[0].cpu()[ok], want_k[ok], dtype)
    assert torch.equal(vp2.view(-1, G * V)[T * (n - 1):T * n], qkv[:, (H + G) * D:])
    # without norms, without rotation
    q = stream.qkv_rotary_prologue(qkv, heads, None, None, 1e-4, POSITIONS.cuda(), None, slots, kp, vp)
    assert torch.equal(q.view(T, -1), qkv[:, :H * D])


@pytest.mark.parametrize("heads,dims", [((4, 32, 16, 64), 16), ((3, 20, 6, 18), 4), ((16, 128, 64, 512), 64),
                                        ((2, 7, 3, 9), 2), ((3, 9, 6, 10), 6)])
@pytest.mark.parametrize("dtype", DT)
def test_latent_prologue_by_halves(heads, dims, dtype):
    from easydel_b200.ops import latent, rotation

    H, D, R, L = heads
    T, ld = 21, H * (D + R) + L + R + 5
    proj = _r(T, ld, dtype=dtype)
    before = proj.clone()
    w = 1 + 0.2 * _r(L, seed=1)
    rot = {"base": 700.0, "dims": dims}
    pages = torch.zeros(3, 128, 1, L + R, dtype=dtype, device="cuda")
    slots = torch.randperm(384, generator=torch.Generator().manual_seed(2))[:T].to(torch.int32).cuda()
    slots[3] = -1
    latent.prologue(proj, heads, w, 1e-5, rotation.pair_frequencies(700.0, dims, "cuda"), POSITIONS.cuda(), slots, pages,
                    "halves")
    _status()
    f = before.cpu().double()
    n = H * (D + R)
    q = f[:, :n].view(T, H, D + R)
    wq = torch.cat([q[..., :D], O.rotate_half(q[..., D:], POSITIONS, rot)], -1)
    row = torch.cat([O.rms_norm(f[:, n:n + L], w.cpu().double(), 1e-5),
                     O.rotate_half(f[:, n + L:n + L + R], POSITIONS, rot)], -1)
    _close(proj[:, :n].cpu(), wq.reshape(T, n), dtype)
    assert torch.equal(proj[:, n:], before[:, n:])
    ok = (slots >= 0).cpu()
    flat = pages.view(384, -1).cpu()
    _close(flat[slots.cpu()[ok].long()], row[ok], dtype)
    assert int((flat.abs().sum(1) > 0).sum()) == T - 1


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,top", [(4, 1), (5, 5), (37, 3), (64, 6), (256, 8), (1000, 32)])
@pytest.mark.parametrize("T", [1, 130, 1500])
def test_softmax_routing_and_tables(E, top, T):
    from easydel_b200.ops.moe_kernels import SoftmaxRouting

    z = 3 * _r(T, E)
    r = SoftmaxRouting(z, top)
    idx, ws = O.route(z.double(), top)
    pos, tok = r.slot_pos.view(T, top).long(), r.row_token
    tiles = int(r.meta[0])
    assert int(r.meta[1]) == tiles * 128 <= r.max_rows and pos.unique().numel() == T * top
    got = r.tile_expert[:tiles].long()[pos // 128]
    assert torch.equal(got.sort(-1).values, idx.sort(-1).values)
    dense = torch.zeros(T, E, dtype=torch.double, device="cuda")
    _close(dense.scatter(1, got, r.weights.double()), dense.scatter(1, idx, ws), torch.float32)
    assert torch.equal(tok[pos], torch.arange(T, device="cuda")[:, None].expand(T, top).to(torch.int32))


@pytest.mark.parametrize("W,F,E,top,shared", [(96, 40, 8, 3, 24), (60, 11, 5, 5, 13), (256, 128, 20, 2, None)])
@pytest.mark.parametrize("T", [1, 700])
@pytest.mark.parametrize("dtype", DT)
def test_experts_with_a_shared_one(W, F, E, top, shared, T, dtype):
    from easydel_b200.layers.moe import MoEBlock
    from easydel_b200.ops import stream

    torch.manual_seed(0)
    blk = MoEBlock(W, F, E, top, scoring="softmax", router_bias=True, shared_intermediate_size=shared or 0, dtype=dtype,
                   init_std=W ** -0.5, expert_init_std=W ** -0.5).cuda()
    blk.gate.bias.copy_(torch.linspace(-1, 1, E))
    h, base = _r(T, W, dtype=dtype), _r(T, W, seed=1)
    w = {"m.router": blk.gate.weight, "m.router.b": blk.gate.bias}
    for e in range(E):
        gu = blk.gate_up_proj.weight[e]
        w.update({f"m.e{e}.gate": gu[:F], f"m.e{e}.up": gu[F:], f"m.e{e}.down": blk.down_proj.weight[e]})
    if shared:
        gu = blk.shared_experts.gate_up_proj.weight
        w.update({"m.shared.gate": gu[:shared], "m.shared.up": gu[shared:],
                  "m.shared.down": blk.shared_experts.down_proj.weight})
    w = {k: v.double() for k, v in w.items()}
    want = O.moe(h.double(), w, "m", O.experts(E, top, F, shared))
    _close(stream.branch_rows(blk.stream_rows(h)), want, dtype, 2)
    got = stream.branch_rows(blk.stream_rows(h, base.clone())).double() - base.double()
    _close(got, want, dtype, 2 if dtype == torch.bfloat16 else 8)
    _status()


# ------------------------------------------------------------------------------------------------ windowed attention
def _layer(scale, window, cap):
    return types.SimpleNamespace(scale=scale, sliding_window=window, softcap=cap, sinks=None)


def _step(shape, layer, lens, new, dtype, spike=(), seed=0, size=1.0):
    """Keys and values of sequences of ``lens`` keys on shuffled pages, queries of their last ``new`` tokens, and what
    attention has to give. ``spike``: key positions (counted back from the sequence's last query) made to stand out."""
    from easydel_b200.caching.paged import PagedBatchMeta, PagedLayerView

    H, G, D, V = shape
    g = torch.Generator().manual_seed(seed)
    per = [-(-n // 128) for n in lens]
    perm = (torch.randperm(sum(per), generator=g) + 1).tolist()
    table = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    kp = torch.full((sum(per) + 1, 128, G, D), 5.0, dtype=dtype)                 # finite filler in unused places
    vp = torch.full((sum(per) + 1, 128, G, V), 5.0, dtype=dtype)
    q = (torch.randn(sum(new), H, D, generator=g) * size).to(dtype)
    want, at = [], 0
    for b, (n, m) in enumerate(zip(lens, new)):
        ids = [perm.pop() for _ in range(per[b])]
        table[b, :per[b]] = torch.tensor(ids)
        k, v = torch.randn(n, G, D, generator=g).to(dtype), torch.randn(n, G, V, generator=g).to(dtype)
        for back in spike:
            if 0 <= n - 1 - back:
                k[n - 1 - back] *= 4
                v[n - 1 - back] *= 4
        for j in range(0, n, 128):
            c = min(128, n - j)
            kp[ids[j // 128], :c], vp[ids[j // 128], :c] = k[j:j + c], v[j:j + c]
        full = torch.cat([torch.zeros(n - m, H, D, dtype=torch.double), q[at:at + m].double()])
        want.append(O.windowed_heads(full, k.double(), v.double(), layer.scale, layer.sliding_window, layer.softcap)[-m:])
        at += m
    cu = torch.tensor([0, *new]).cumsum(0).to(torch.int32).cuda()
    meta = PagedBatchMeta(cu_q=cu, kv_lens=_i32(*lens), page_table=table.cuda(), slot_mapping=None, max_q=max(new),
                          num_seqs=len(lens), spans=list(zip(new, lens)))
    return q.cuda(), PagedLayerView(kp.cuda(), vp.cuda()), meta, torch.cat(want).cuda()


SHAPES = [(6, 2, 48, 24), (16, 2, 128, 64), (34, 2, 64, 128), (3, 1, 20, 12), (4, 4, 16, 40), (1, 1, 8, 8), (6, 2, 96, 96),
          (4, 1, 136, 72)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,cap", [(None, 3.0), (1, 2.0), (44, 4.0), (128, 0.0), (300, 2.5)])
@pytest.mark.parametrize("dtype", DT)
def test_windowed_attention_decode(shape, window, cap, dtype):
    layer = _layer(shape[2] ** -0.5, window, cap)
    edge = (window or 1) - 1
    lens = [1, 31, 44, 45, 128, 129, 300, 301, 517]
    q, view, meta, want = _step(shape, layer, lens, [1] * len(lens), dtype, spike=(edge, edge + 1))
    for splits in (1, 3):
        meta.num_splits = splits
        got = view.attend_pages(layer, q, meta)
        _status()
        _close(got, want, dtype, 2.5)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window,cap", [(None, 3.0), (1, 2.0), (44, 4.0), (129, 0.0), (300, 2.5)])
@pytest.mark.parametrize("dtype", DT)
def test_windowed_attention_portions_beside_single_tokens(shape, window, cap, dtype):
    layer = _layer(shape[2] ** -0.5, window, cap)
    edge = (window or 1) - 1
    new, lens = [1, 1, 2, 130, 257, 3, 1, 64], [5, 290, 400, 130, 400, 129, 260, 64]
    q, view, meta, want = _step(shape, layer, lens, new, dtype, spike=(edge, edge + 1, 127, 128))
    got = view.attend_pages(layer, q, meta)
    _status()
    _close(got, want, dtype, 2.5)


@pytest.mark.parametrize("size,cap", [(1.0, 10.0), (6.0, 10.0), (8.0, 60.0), (14.0, 60.0), (30.0, 200.0), (90.0, 200.0)])
@pytest.mark.parametrize("new", [1, 200])
def test_cap_of_16_bit_heads_is_computed_in_32_bits(size, cap, new):
    """Scores from well below the cap to far above it; under the large cap a score's last 16-bit digit would be a tenth."""
    shape = (4, 2, 64, 64)
    layer = _layer(64 ** -0.5, 150, cap)
    q, view, meta, want = _step(shape, layer, [260, 300], [new, new], torch.bfloat16, size=size)
    _close(view.attend_pages(layer, q, meta), want, torch.bfloat16, 2.5)
    _status()


def test_window_edges_are_seen_and_not_seen():
    """One key stands far above the rest: a query whose window just holds it copies its value, the next one does not."""
    from easydel_b200.caching.paged import PagedLayerView

    n, H, G, D = 420, 4, 2, 64
    for dtype in DT:
        for window in (16, 128, 200):
            layer = _layer(1.0, window, 60.0)
            q, view, meta, _ = _step((H, G, D, D), layer, [n], [n], dtype)
            ids = meta.page_table[0, :4].long()
            q = torch.zeros_like(q)
            q[..., 0] = 8.0
            for key in (0, 1, 127, 128, 190):
                kp = torch.zeros_like(view.k_pages)
                kp[ids[key // 128], key % 128, :, 0] = 8.0        # 64 before the cap, 47 after it; the others have 0
                got = PagedLayerView(kp, view.v_pages).attend_pages(layer, q, meta)
                value = view.v_pages[ids[key // 128], key % 128].double().repeat_interleave(H // G, 0)
                err = ((got.double() - value).abs().amax((1, 2)) / value.abs().max()).tolist()
                for i in range(n):
                    assert (err[i] < 0.02) == (0 <= i - key < window), (dtype, window, key, i, err[i])
    _status()


# ------------------------------------------------------------------------------------------------ latent attention
@pytest.mark.parametrize("dtype", DT)
def test_far_keys_and_sinks_of_latent_layers(tmp_path, dtype):
    """A latent layer alone finds one token far back, in a prompt and in decoding, and its sink takes a share."""
    cfg = O.random_config([O.latent(4, 16, 32, 32, 64, 0.4, base=1e6)], 64, 96, mult=1.0, embed_scale=1.0)
    w = O.random_weights(cfg, 1)
    w["l0.mix.q"] = (w["l0.mix.q"].float() * 3).to(torch.bfloat16)
    cfg, w, model = C.make(tmp_path, "far", dtype, "cuda", cfg=cfg, weights=w)
    toks = C.tokens(420, 96, 3)
    want = O.forward(cfg, w, toks)
    assert C.error(O.forward(cfg, w, toks, mutate="no_sink"), want) > 0.1
    floor = 2e-5 if dtype == torch.float32 else 2 * C.bf16_floor(cfg, w, toks)
    for cuts in ([420], [300, 1], [129, 2, 64]):
        assert C.error(C.run_cut(C.replayer(model), "a", toks, cuts), want) < floor


# ------------------------------------------------------------------------------------------------ whole models
def _quantile(got, want, q):
    d = got.double() - want.double()
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).quantile(q))


def _check(cfg, w, got, toks, dtype):
    want = O.forward(cfg, w, toks)
    if dtype == torch.float32:
        assert C.error(got, want) < 3e-5
        return
    rough = O.forward(cfg, w, toks, dtype=torch.bfloat16)      # a few rows may choose other experts in 16 bits
    assert _quantile(got, want, 0.8) < 1.5 * _quantile(rough, want, 0.8), (_quantile(got, want, 0.8),
                                                                           _quantile(rough, want, 0.8))


@pytest.mark.parametrize("name", sorted(C.CONFIGS))
@pytest.mark.parametrize("cuts", [[400], [370, 1], [2, 3, 1, 129, 64]])
@pytest.mark.parametrize("dtype", DT)
def test_models_in_portions_and_decoding(tmp_path, name, cuts, dtype):
    cfg, w, model = C.make(tmp_path, name, dtype, "cuda")
    toks = C.tokens(400, cfg["vocab"], 3)
    rep = C.replayer(model)
    assert rep.engine.runner.use_graphs
    _check(cfg, w, C.run_cut(rep, "a", toks, cuts), toks, dtype)


@pytest.mark.parametrize("name", ["mixed", "wide"])
@pytest.mark.parametrize("dtype", DT)
def test_mixed_batches_reuse_pages(tmp_path, name, dtype):
    cfg, w, model = C.make(tmp_path, name, dtype, "cuda")
    rep = C.replayer(model, max_tokens=768, max_requests=3)
    pool_free = [m.pool.num_free for m in rep.engine.kv.managers]
    seqs = {n: C.tokens(k, cfg["vocab"], i) for i, (n, k) in enumerate(
        [("a", 300), ("b", 5), ("c", 90), ("d", 259), ("e", 2)])}
    got, at = {n: [] for n in seqs}, {n: 0 for n in seqs}
    plan = [[("a", 200), ("b", 1)], [("a", 98), ("b", 2), ("c", 64)], [("b", 2), ("a", 1)], [("a", 1), ("c", 1), ("d", 230)],
            [("d", 2), ("c", 25), ("e", 1)], [("d", 26), ("e", 1)], [("d", 1)]]
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
        if len(toks) > 50 or dtype == torch.float32:
            _check(cfg, w, torch.cat(got[n]), toks, dtype)
    assert [m.pool.num_free for m in rep.engine.kv.managers] == pool_free


@pytest.mark.parametrize("dtype", DT)
def test_cuts_and_company_do_not_matter(tmp_path, dtype):
    """The same tokens whole, in portions and beside other requests: equal beyond rounding."""
    cfg = O.random_config([O.windowed(4, 2, 64, 64, 0.1, 60, 8.0, mlp=O.dense(128)),
                           O.latent(8, 32, 16, 32, 64, 0.15, mlp=O.dense(96)),
                           O.windowed(8, 2, 32, 128, 0.15, 200, 8.0, dims=16, mlp=O.dense(64))], 128, 96)
    cfg, w, model = C.make(tmp_path, "dense", dtype, "cuda", cfg=cfg)
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
    assert C.error(whole, O.forward(cfg, w, toks)) < floor


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
    eng = eSurge(model, max_model_len=512, max_num_seqs=4, num_pages=16)
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (5, 300, 64)]
    sp = SamplingParams(max_tokens=140, temperature=0.0, ignore_eos=True)
    first = [o.outputs[0].token_ids for o in eng.generate(prompts, sp)]
    assert [len(t) for t in first] == [140] * 3
    # every generated token is (nearly) the best one of the plain form given the tokens before it
    for p, t in zip(prompts, first):
        lg = O.forward(cfg, w, p + t)[len(p) - 1:-1]
        gap = (lg.max(-1).values - lg.gather(1, torch.tensor(t)[:, None])[:, 0]) / lg.std()
        assert float(gap.quantile(0.95)) < 0.3
    _status()
