"""Disunex on the GPU: every kernel of the family against plain forms, whole models against a plain restatement."""

import math

import disunex_cases as C
import oracle_disunex as O
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
@pytest.mark.parametrize("W", [60, 77, 352, 1024, 3000, 8192, 9000])
@pytest.mark.parametrize("dtype", DT)
def test_norm_after_the_sum(W, dtype):
    from easydel_b200.ops import stream
    from easydel_b200.ops.moe_kernels import ExpertRows

    x, y, w = 3 * _r(37, W), _r(37, W, seed=1), 0.3 * _r(W, seed=2)
    want = O.norm_after_sum(x.double(), y.double(), 1.7, w.double(), 1e-5)
    s, h = stream.post_norm(x.clone(), y, 1.7, w, 1e-5, dtype, 1.0)
    _close(s, want, torch.float32)
    _close(h, want, dtype)
    # the branch as weighted expert rows, some of them nobody's
    ys, wts = _r(200, W, seed=3, dtype=dtype), torch.rand(37, 3).cuda()
    pos = torch.randint(0, 200, (37, 3), generator=torch.Generator().manual_seed(4)).to(torch.int32).cuda()
    pos[5, 1] = -1
    rows = ExpertRows(ys, wts, pos.reshape(-1).contiguous())
    branch = (ys.double()[pos.clamp_min(0).long()] * (wts * (pos >= 0)).double()[..., None]).sum(1)
    s, h = stream.post_norm(x.clone(), rows, 0.5, w, 1e-5, dtype, 1.0)
    _close(s, O.norm_after_sum(x.double(), branch, 0.5, w.double(), 1e-5), torch.float32)
    plain = stream.norm_shift(x, w, 1e-5, dtype, offset=1.0)
    _close(plain, O.rms_norm(x, 1 + w, 1e-5), dtype)
    many = stream.norm_shift(x.repeat(70, 1), w, 1e-5, dtype, offset=1.0)       # the form that walks several rows
    assert torch.equal(many[-37:], many[:37])
    _close(many[:37], O.rms_norm(x, 1 + w, 1e-5), dtype)


@pytest.mark.parametrize("dtype", DT)
def test_gelu_and_head_gate(dtype):
    from easydel_b200.ops import latent, stream

    for n in (41, 64):
        z = 3 * _r(37, n, dtype=dtype)
        _close(stream.gelu_erf(z), O.gelu_erf(z.double()), dtype)
    for H, V in ((3, 12), (4, 64), (5, 7)):
        o, g = _r(H, 19, V, dtype=dtype), 2 * _r(19, 30 + H * V, seed=1, dtype=dtype)
        out = torch.empty(19, H * V, dtype=dtype, device="cuda")
        gate = g[:, 30:] if H != 4 else g[:, 24:24 + H * V]
        latent.head_gate(o.transpose(0, 1), gate, out)
        _close(out, o.transpose(0, 1).reshape(19, H * V).double() * O.sigmoid(gate.double()), dtype)


@pytest.mark.parametrize("heads,dims", [((4, 32, 16, 64), 16), ((3, 20, 6, 18), 4), ((16, 128, 64, 512), 64),
                                        ((2, 7, 3, 9), 2)])
@pytest.mark.parametrize("dtype", DT)
def test_prologue(heads, dims, dtype):
    """Rotated queries in place, cache rows on their pages; at positions far beyond any table too."""
    from easydel_b200.ops import latent, rotation

    H, D, R, L = heads
    T, ld = 21, H * (D + R) + L + R + 5
    proj = _r(T, ld, dtype=dtype)
    before = proj.clone()
    w = 1 + 0.2 * _r(L, seed=1)
    pos = torch.tensor([*range(11), *range(1000, 1005), 30001, 99999, 100000, 100001, 250000], dtype=torch.int32)
    freq = rotation.pair_frequencies(700.0, dims, "cuda")
    pages = torch.zeros(3, 128, 1, L + R, dtype=dtype, device="cuda")
    slots = torch.randperm(384, generator=torch.Generator().manual_seed(2))[:T].to(torch.int32).cuda()
    slots[3] = -1
    latent.prologue(proj, heads, w, 1e-5, freq, pos.cuda(), slots, pages)
    _status()
    f = before.cpu().double()
    n = H * (D + R)
    q = f[:, :n].view(T, H, D + R)
    wq = torch.cat([q[..., :D], O.rotate_pairs(q[..., D:], pos, 700.0, dims)], -1)
    row = torch.cat([O.rms_norm(f[:, n:n + L], w.cpu().double(), 1e-5),
                     O.rotate_pairs(f[:, n + L:n + L + R], pos, 700.0, dims)], -1)
    _close(proj[:, :n].cpu(), wq.reshape(T, n), dtype)
    assert torch.equal(proj[:, n:], before[:, n:])
    assert torch.equal(proj[:, :n].view(T, H, D + R)[..., :D], before[:, :n].view(T, H, D + R)[..., :D])
    ok = (slots >= 0).cpu()
    flat = pages.view(384, -1).cpu()
    _close(flat[slots.cpu()[ok].long()], row[ok], dtype)
    assert int((flat.abs().sum(1) > 0).sum()) == T - 1


# ------------------------------------------------------------------------------------------------ experts
@pytest.mark.parametrize("E,top", [(4, 1), (20, 2), (37, 5), (64, 6), (100, 8), (256, 8), (1000, 32)])
@pytest.mark.parametrize("T", [1, 9, 130, 1500])
def test_routing_and_tables(E, top, T):
    from easydel_b200.ops.moe_kernels import SigmoidRouting

    z, corr = 2 * _r(T, E), 0.4 * _r(E, seed=1)
    r = SigmoidRouting(z, corr, top)
    idx, ws = O.route(z.double(), corr.double(), top)
    pos, tok = r.slot_pos.view(T, top).long(), r.row_token
    tiles = int(r.meta[0])
    assert int(r.meta[1]) == tiles * 128 <= r.max_rows and pos.unique().numel() == T * top
    got = r.tile_expert[:tiles].long()[pos // 128]
    assert torch.equal(got.sort(-1).values, idx.sort(-1).values)
    dense = torch.zeros(T, E, dtype=torch.double, device="cuda")
    _close(dense.scatter(1, got, r.weights.double()), dense.scatter(1, idx, ws), torch.float32)
    assert torch.equal(tok[pos], torch.arange(T, device="cuda")[:, None].expand(T, top).to(torch.int32))
    assert int((tok[:tiles * 128] >= 0).sum()) == T * top


@pytest.mark.parametrize("W,F,E,top", [(96, 40, 8, 3), (60, 11, 37, 5), (256, 128, 20, 2)])
@pytest.mark.parametrize("T", [1, 33, 700])
@pytest.mark.parametrize("dtype", DT)
def test_clamped_experts(W, F, E, top, T, dtype):
    from easydel_b200.ops.moe_kernels import SigmoidRouting, clamped_experts

    h, z = _r(T, W, dtype=dtype), _r(T, E, seed=1)
    gu, dn = 2 * _r(E, 2 * F, W, seed=2, dtype=dtype) / W ** 0.5, _r(E, W, F, seed=3, dtype=dtype) / F ** 0.5
    w = {f"m.e{e}.{n}": t.double() for e in range(E) for n, t in (("gate", gu[e, :F]), ("up", gu[e, F:]), ("down", dn[e]))}
    w["m.router"], w["m.correction"] = torch.eye(E).double().cuda(), torch.zeros(E).double().cuda()
    got = clamped_experts(h, SigmoidRouting(z, None, top), gu, dn, 0.8).combine()
    idx, ws = O.route(z.double(), 0.0, top)
    want = torch.zeros(T, W, dtype=torch.double, device="cuda")
    for e in range(E):
        t, k = (idx == e).nonzero(as_tuple=True)
        want[t] += ws[t, k][:, None] * O.clamped_expert(h[t].double(), w, f"m.e{e}", 0.8)
    _close(got, want, dtype, 2)
    _status()


# ------------------------------------------------------------------------------------------------ attention
def _layer(H, D, R, V, L, dtype, window, seed=0):
    from easydel_b200.layers.mla import LatentStreamAttention

    torch.manual_seed(seed)
    a = LatentStreamAttention(64, H, dim=D, rot_dim=R, vdim=V, kv_rank=L, scale=(D + R) ** -0.5, sliding_window=window,
                              use_sinks=True, output_gate=True, dtype=dtype, init_std=L ** -0.5).cuda()
    a.sinks.copy_(torch.linspace(-1.5, 2.5, H))
    return a


def _step(a, lens, new, dtype, spike=(), seed=0):
    """Cache rows of sequences of ``lens`` keys on shuffled pages, projected rows of their last ``new`` tokens, and what
    attention has to give. ``spike``: key positions (counted back from the sequence's last query) made to stand out."""
    from easydel_b200.caching.paged import PagedBatchMeta

    g = torch.Generator().manual_seed(seed)
    H, D, R, V, L = a.heads, a.dim, a.rot_dim, a.vdim, a.kv_rank
    per = [-(-n // 128) for n in lens]
    perm = (torch.randperm(sum(per), generator=g) + 1).tolist()
    table = torch.zeros(len(lens), max(per) + 1, dtype=torch.int32)
    pages = torch.full((sum(per) + 1, 128, 1, L + R), 5.0, dtype=dtype)          # finite filler in unused places
    proj = torch.randn(sum(new), H * (D + R) + L + R + H * V, generator=g).to(dtype)
    up = a.ukv_proj.weight.detach().cpu().double()
    uk, uv = up[:H * D].view(H, D, L), up[H * D:].view(H, V, L)
    want, at = [], 0
    for b, (n, m) in enumerate(zip(lens, new)):
        ids = [perm.pop() for _ in range(per[b])]
        table[b, :per[b]] = torch.tensor(ids)
        rows = torch.randn(n, L + R, generator=g).to(dtype)
        for back in spike:
            if 0 <= n - 1 - back:
                rows[n - 1 - back] *= 4
        for j in range(n):
            pages[ids[j // 128], j % 128, 0] = rows[j]
        q = proj[at:at + m, :H * (D + R)].view(m, H, D + R).double()
        full = torch.cat([torch.zeros(n - m, H, D + R, dtype=torch.double), q])
        o = O.latent_heads(full, rows[:, :L].double(), rows[:, L:].double(), uk, uv, D, a.scale, a.sliding_window,
                           a.sinks.cpu().double())[-m:]
        want.append(o.reshape(m, H * V) * O.sigmoid(proj[at:at + m, -H * V:].double()))
        at += m
    cu = torch.tensor([0, *new]).cumsum(0).to(torch.int32).cuda()
    meta = PagedBatchMeta(cu_q=cu, kv_lens=_i32(*lens), page_table=table.cuda(), slot_mapping=None, max_q=max(new),
                          num_seqs=len(lens), spans=list(zip(new, lens)))
    return proj.cuda(), pages.cuda(), meta, torch.cat(want).cuda()


SHAPES = [(4, 32, 16, 48, 64), (16, 64, 64, 64, 256), (17, 128, 64, 128, 512), (6, 56, 16, 64, 136), (3, 20, 6, 12, 18),
          (5, 96, 24, 72, 456), (2, 128, 0, 128, 64), (1, 8, 8, 8, 8)]


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [None, 1, 44, 128, 300])
@pytest.mark.parametrize("dtype", DT)
def test_latent_attention_decode(shape, window, dtype):
    from easydel_b200.ops import latent

    a = _layer(*shape, dtype, window)
    edge = (window or 1) - 1
    lens = [1, 31, 44, 45, 128, 129, 300, 301, 517]
    proj, pages, meta, want = _step(a, lens, [1] * len(lens), dtype, spike=(edge, edge + 1))
    got = latent.attend(a, proj, pages, meta, meta.page_table)
    _status()
    _close(got, want, dtype, 2.5)


@pytest.mark.parametrize("splits", [2, 3, 8])
@pytest.mark.parametrize("window", [0, 200])
def test_latent_decode_with_key_splits(splits, window):
    from easydel_b200.ops import serving as S

    a = _layer(17, 128, 64, 128, 512, torch.bfloat16, window or None)
    proj, pages, meta, want = _step(a, [700, 3, 260], [1, 1, 1], torch.bfloat16, spike=(199, 200))
    up = a.ukv_proj.weight
    q = proj[:, :17 * 192].view(3, 17, 192)
    ql = torch.einsum("bhd,hdl->bhl", q[..., :128], up[:17 * 128].view(17, 128, 512))
    o = S.latent_decode(ql, q[..., 128:], pages, meta.kv_lens, meta.page_table, scale=a.scale, window=window,
                        sinks=a.sinks, num_splits=splits)
    o = torch.einsum("bhl,hvl->bhv", o.float(), up[17 * 128:].view(17, 128, 512).float()).reshape(3, -1)
    _status()
    _close(o * torch.sigmoid(proj[:, -17 * 128:].float()), want, torch.bfloat16, 2.5)


@pytest.mark.parametrize("shape", SHAPES)
@pytest.mark.parametrize("window", [None, 1, 44, 129, 300])
@pytest.mark.parametrize("dtype", DT)
def test_latent_attention_portions_beside_single_tokens(shape, window, dtype):
    from easydel_b200.ops import latent

    a = _layer(*shape, dtype, window)
    edge = (window or 1) - 1
    new = [1, 1, 2, 130, 257, 3, 1, 64]
    lens = [5, 290, 400, 130, 700, 129, 260, 64]
    proj, pages, meta, want = _step(a, lens, new, dtype, spike=(edge, edge + 1, 127, 128))
    got = latent.attend(a, proj, pages, meta, meta.page_table)
    _status()
    _close(got, want, dtype, 2.5)


def test_window_edges_are_seen_and_not_seen():
    """One key stands far above the rest: a query whose window just holds it copies its value, the next one does not."""
    from easydel_b200.ops import latent

    for dtype in DT:
        for window in (16, 128, 200):
            a = _layer(2, 64, 16, 64, 64, dtype, window)
            a.sinks.fill_(-1e4)
            n = 420
            proj, pages, meta, _ = _step(a, [n], [n], dtype)
            H, D, R, L = 2, 64, 16, 64
            flat = pages[meta.page_table[0, :4].long()].view(-1, L + R)
            for key in (0, 1, 127, 128, 190):
                f = flat.clone()
                f[:, L:] = 0
                f[key, L] = 30.0                                  # only this key has a rotary part
                p = proj.clone()
                p[:, :H * (D + R)] = 0
                p[:, D], p[:, D + R + D] = 30.0, 30.0             # every query asks for it
                pg = torch.zeros_like(pages)
                pg[meta.page_table[0, :4].long()] = f.view(4, 128, 1, L + R)
                meta.visible.clear()
                got = latent.attend(a, p, pg, meta, meta.page_table).view(n, 2, 64)
                up = a.ukv_proj.weight[H * D:].view(2, 64, L).double()
                value = torch.einsum("hvl,l->hv", up, f[key, :L].double())
                gate = O.sigmoid(p[:, -128:].double()).view(n, 2, 64)
                err = ((got.double() - value * gate).abs().amax((1, 2)) / value.abs().max()).tolist()
                for i in range(n):
                    inside = 0 <= i - key < window
                    assert (err[i] < 0.02) == inside, (dtype, window, key, i, err[i])
    _status()


# ------------------------------------------------------------------------------------------------ whole models
def _quantile(got, want, q=0.9):
    d = got.double() - want.double()
    return float((d.pow(2).mean(-1).sqrt() / want.double().std()).quantile(q))


def _check(cfg, w, got, toks, dtype):
    want = O.forward(cfg, w, toks)
    if dtype == torch.float32:
        assert C.error(got, want) < 2e-5
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


@pytest.mark.parametrize("name", ["shared", "wide"])
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
    cfg = O.random_config([O.latent(4, 64, 32, 64, 128, 0.1, window=60, mlp=O.dense(128)),
                           O.latent(8, 32, 16, 32, 64, 0.15, window=200, mlp=O.dense(96))], 128, 96, alpha=2.0)
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

    cfg, w, model = C.make(tmp_path, "shared", torch.float32, "cuda")
    prompts = [C.tokens(n, cfg["vocab"], n) for n in (1, 13, 200, 40)]
    eng = eSurge(model, max_model_len=256, max_num_seqs=3, num_pages=5, max_num_batched_tokens=48)
    outs = eng.generate(prompts, SamplingParams(max_tokens=8, temperature=0.0, ignore_eos=True))
    for p, o in zip(prompts, outs):
        assert o.outputs[0].token_ids == C.greedy(cfg, w, p, 8)
    assert eng.runner.timings["graph_steps"] > 0
    _status()


def test_16_bit_generation_serves_and_repeats(tmp_path):
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
    assert math.isfinite(sum(sum(t) for t in first))
    _status()
