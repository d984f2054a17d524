"""The Zetonex design in the engine against its plain statement (tests/plain_zetonex.py): the new kernels alone, each
mechanism alone in a model, then whole models in every way of cutting the work (whole prompts, a decoded tail, portions
down to two tokens, mixed batches with pages used again), keys at the edges of windows, kept positions and pages and far back,
long decoding through captured graphs, and greedy generation through the entry point and its scheduler. Cache pages are
poisoned with NaN so that a read outside a request's own rows shows."""
import random

import numpy as np
import pytest
import torch

import helpers
import plain_zetonex as plain
import zetonex_helpers as zh

pytestmark = pytest.mark.gpu

TOL = {"float32": 5e-5, "bfloat16": 4e-2}     # relative to the largest |logit| of the plain statement
LENGTHS = [1, 7, 33, 90, 61, 47, 2, 70, 18, 120, 64, 65, 3]


def row_errors(got, want):
    scale = max(float(np.abs(w).max()) for w in want.values())
    return np.array([float(np.abs(got[r][p].astype(np.float64) - want[r][p]).max()) / scale
                     for r in sorted(got) for p in sorted(got[r])])


def agrees(got, want, dtype):
    """float32: every row within the tolerance; this is what judges the cache and the batching. bfloat16: activations rounded
    to 8 bits through several layers (and a difference of two rounded maps divided by its own size) leave a few rows further off
    than the typical row, so nearly all rows must be within the tolerance, the typical row well within it, and none far
    outside."""
    err = row_errors(got, want)
    if not np.isfinite(err).all():
        return False
    if dtype == "float32":
        return bool(err.max() <= TOL[dtype])
    return bool((err > TOL[dtype]).mean() <= 0.05 and np.median(err) <= TOL[dtype] / 2 and err.max() <= 6 * TOL[dtype])


def run(folder, dtype, steps, page, **kw):
    from tinyinfer_b200.engine.replay import TraceSession
    session = TraceSession(folder, dtype, helpers.peak_tokens(steps, max(64, page)), page_size=page, poison_cache=True, **kw)
    got = helpers.collect(session, steps)
    session.runner.check_status()
    session.runner.manager.check_consistency()
    return got, session


def ints(values):
    return torch.tensor(values, dtype=torch.int32).cuda()


def paged(lens, page, gen):
    """A shuffled block table for requests of these lengths, and the number of pages of the pool."""
    counts = [(n + page - 1) // page for n in lens]
    perm = torch.randperm(sum(counts) + 3, generator=gen).tolist()
    table, at = [], 0
    for c in counts:
        table.append(perm[at:at + c] + [-1] * (max(counts) - c))
        at += c
    return torch.tensor(table, dtype=torch.int32), sum(counts) + 3


# ------------------------------------------------------------------ the kernels alone
@pytest.mark.parametrize("hq,hkv,d,dv,maps,v_is_k,rot,norm", [
    (6, 2, 10, 28, 2, False, 6, True), (4, 2, 32, 64, 2, False, 16, True), (2, 1, 64, 128, 2, False, 64, True),
    (3, 3, 7, 14, 2, False, 0, True), (6, 3, 20, 20, 1, True, 12, False), (4, 2, 64, 64, 1, True, 32, False),
    (16, 8, 128, 128, 1, True, 64, False), (1, 1, 5, 5, 1, True, 0, False), (16, 8, 64, 128, 2, False, 64, True)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_head_preparation_against_plain(hq, hkv, d, dv, maps, v_is_k, rot, norm, dtype):
    """Norm and rotation per map, values that are the keys before both, and every key and value where its page says."""
    from tinyinfer_b200 import ops
    from tinyinfer_b200.config import PositionSpec
    from tinyinfer_b200.parts.base import build_position
    gen = torch.Generator().manual_seed(hq * d + maps)
    lens, page, pad, kd = [37, 1, 90], 8, 8, maps * d
    nq, nk, nv = hq * kd, hkv * kd, 0 if v_is_k else hkv * dv
    table, pages = paged(lens, page, gen)
    planes = kd == dv
    cache = torch.full((2, pages, hkv, page, kd) if planes else (1, pages, hkv, page, kd + dv), float("nan"), dtype=dtype).cuda()
    rows = torch.randn(sum(lens), pad + nq + nk + nv + 3, generator=gen).to(dtype)
    wq, wk = (1 + 0.3 * torch.randn(d, generator=gen) for _ in range(2)) if norm else (None, None)
    rotation = build_position(PositionSpec(kind="rope", theta=777.0, rotary_dim=rot, exact_frequencies=True) if rot else
                              PositionSpec(kind="none"), dtype, "cuda").rotation()
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    q = ops.head_rotation(rows.cuda(), num_heads=hq, num_kv_heads=hkv, head_dim=d, v_dim=dv, has_kv=True, offset=pad,
                          positions=ints([p for n in lens for p in range(n)]), token_seq=ints([i for i, n in enumerate(lens) for _ in range(n)]),
                          q_norm_weight=wq.cuda() if norm else None, k_norm_weight=wk.cuda() if norm else None, eps=1e-5,
                          rotation=rotation, cache=cache, block_table=table.cuda(), status=status, maps=maps, values_are_keys=v_is_k)
    assert int(status.item()) == 0 and tuple(q.shape) == (sum(lens), hq, kd)
    q, cache, at = q.cpu().double(), cache.cpu().double(), 0
    tol = 5e-5 if dtype == torch.float32 else 1.2e-2
    for i, n in enumerate(lens):
        x = rows[at:at + n, pad:].double()
        heads = {"q": x[:, :nq].reshape(n, hq * maps, d), "k": x[:, nq:nq + nk].reshape(n, hkv * maps, d)}
        v = heads["k"] if v_is_k else x[:, nq + nk:nq + nk + nv].reshape(n, hkv, dv)
        for name, w in (("q", wq), ("k", wk)):
            y = plain.rms(heads[name], 1e-5) * w.double() if norm else heads[name]
            heads[name] = plain.rotated(y, dict(base=777.0, dims=rot)).reshape(n, -1, kd)
        assert (q[at:at + n] - heads["q"]).abs().max() <= tol * max(1.0, heads["q"].abs().max()), i
        for p in range(n):
            slot = cache[:, table[i, p // page], :, p % page]
            gk, gv = (slot[0], slot[1]) if planes else (slot[0, :, :kd], slot[0, :, kd:])
            assert (gk - heads["k"][p]).abs().max() <= tol * max(1.0, heads["k"].abs().max()), (i, p)
            assert torch.equal(gv, v[p]), (i, p)          # not touched, not rounded again
        at += n


SHAPES = [
    # hq, hkv, features of a key (all maps), dv, page, [(context, q_len)]
    (6, 2, 20, 28, 8, [(37, 37), (50, 1), (9, 2)]),                       # rows of [k | v]: the float32-arithmetic kernel
    (3, 1, 8, 40, 4, [(130, 1), (17, 17)]),
    (6, 3, 80, 80, 16, [(150, 150), (131, 1), (90, 3)]),                  # two planes, a size the tensor-core kernels refuse
    (8, 2, 64, 64, 16, [(130, 130), (129, 1), (200, 2)]),                 # two planes: the tensor-core kernels
    (8, 4, 128, 128, 64, [(1500, 1), (1, 1), (256, 1), (257, 1), (700, 513)]),
    (4, 4, 128, 128, 64, [(1300, 897), (64, 64), (65, 1), (390, 130)]),
    (6, 2, 64, 64, 32, [(600, 600), (131, 1), (90, 3)]),
    (8, 1, 128, 128, 16, [(2400, 200), (2560, 1), (2561, 1), (640, 384)]),
]


def attention_case(work, page, hq, hkv, kd, dv, dtype, window, keep, gen, loud=2.0):
    """Queries, a cache whose every row that no query of the step may read is NaN (pages given back, never written), tables."""
    lens = [c for c, _ in work]
    table, total = paged(lens, page, gen)
    planes = kd == dv
    cache = torch.full((2, total, hkv, page, kd) if planes else (1, total, hkv, page, kd + dv), float("nan"), dtype=dtype)
    ks = [torch.randn(n, hkv, kd, generator=gen).to(dtype) for n in lens]
    vs = [torch.randn(n, hkv, dv, generator=gen).to(dtype) for n in lens]
    for i, (n, q_len) in enumerate(work):
        lo = max(0, n - q_len - (window or n) + 1)
        held = {p // page for p in range(n) if p >= lo or p < keep}
        for p in range(n):
            if p // page not in held:
                continue
            pg = table[i, p // page]
            if planes:
                cache[0, pg, :, p % page], cache[1, pg, :, p % page] = ks[i][p], vs[i][p]
            else:
                cache[0, pg, :, p % page] = torch.cat([ks[i][p], vs[i][p]], dim=-1)
        for j in range(table.shape[1]):
            if j not in held:
                table[i, j] = -1
    pos = torch.tensor([p for c, n in work for p in range(c - n, c)], dtype=torch.int32)
    seq = torch.tensor([i for i, (c, n) in enumerate(work) for _ in range(n)], dtype=torch.int32)
    q = (loud * torch.randn(pos.shape[0], hq, kd, generator=gen)).to(dtype)
    return q, cache, ks, vs, table, pos, seq


def attend(q, cache, dv, planes, table, pos, seq, **kw):
    from tinyinfer_b200 import ops
    status = torch.zeros(1, dtype=torch.int32, device="cuda")
    args = dict(positions=pos.cuda(), token_seq=seq.cuda(), block_table=table.cuda(), status=status, **kw)
    out = ops.paged_attention(q.cuda(), cache.cuda(), **args) if planes else ops.attention_rows(q.cuda(), cache.cuda(), v_dim=dv, **args)
    assert int(status.item()) == 0
    ops.check_kernel_status()
    return out.cpu().double()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("pairs", [False, True])
@pytest.mark.parametrize("window,keep,gate,softcap", [
    (1, 1, True, None), (7, 3, True, None), (64, 64, False, None), (110, 4, True, None), (129, 200, True, 4.0), (300, 16, False, None),
    (65, 129, True, None), (200, 0, True, None), (40, 700, False, 4.0)])
@pytest.mark.parametrize("hq,hkv,d,dv,page,work", SHAPES)
def test_attention_with_kept_positions_and_gates(monkeypatch, dtype, pairs, window, keep, gate, softcap, hq, hkv, d, dv, page, work):
    """Windows and kept positions smaller and larger than the kernels' tiles and pages, on their borders and off them, apart
    and overlapping, in every attention kernel, with and without a gate per feature."""
    from tinyinfer_b200 import ops
    if pairs and (d != dv or d not in (64, 128) or dtype == torch.float32):
        pytest.skip("one form of the prompt kernel")
    monkeypatch.setattr(ops, "PAIR_MIN_CTAS", 0 if pairs else 1 << 30)
    gen = torch.Generator().manual_seed(hq * d + window)
    q, cache, ks, vs, table, pos, seq = attention_case(work, page, hq, hkv, d, dv, dtype, window, keep, gen)
    T = q.shape[0]
    logits = torch.randn(T, 8 + hq * dv + (-hq * dv) % 8, generator=gen).to(dtype)
    extras = dict(gate=logits.cuda(), gate_offset=8, feature_gate=True) if gate else {}
    scale = d ** -0.5
    out = attend(q, cache, dv, d == dv, table, pos, seq, scale=scale, window=window, keep_first=keep, softcap=softcap or 0.0, **extras)
    want, at = [], 0
    for i, (n, q_len) in enumerate(work):
        mask = plain.seen(n, window, keep)[n - q_len:]
        for h in range(hq):
            g = h * hkv // hq
            p = plain.softmax_weights(q[at:at + q_len, h].double(), ks[i][:, g].double(), scale, mask, softcap)
            want.append((slice(at, at + q_len), h, p @ vs[i][:, g].double()))
        at += q_len
    worst = 0.0
    for rows, h, o in want:
        if gate:
            o = o * torch.sigmoid(logits[rows, 8 + h * dv:8 + (h + 1) * dv].double())
        worst = max(worst, float((out[rows, h * dv:(h + 1) * dv] - o).abs().max()))
    assert worst <= (2e-5 if dtype == torch.float32 else 3e-2), worst


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("window,keep,softcap", [(None, 0, None), (1, 0, 3.0), (33, 0, None), (128, 0, 3.0), (129, 0, None), (500, 0, 3.0),
                                                 (50, 20, None), (70, 300, 3.0)])
@pytest.mark.parametrize("hq,hkv,d,dv,page,work", SHAPES)
def test_differential_attention_against_plain(dtype, window, keep, softcap, hq, hkv, d, dv, page, work):
    """Two maps a head over one value, in every attention kernel: windows on and off the borders of tiles, contexts that one
    CTA and that several share, prompts of one and of many query tiles, a gate behind the norm."""
    gen = torch.Generator().manual_seed(hq * d + (window or 0))
    q, cache, ks, vs, table, pos, seq = attention_case(work, page, hq, hkv, d, dv, dtype, window, keep, gen)
    half, share, eps, factor, scale = d // 2, 0.4, 1e-5, 0.7, (d // 2) ** -0.5
    logits = torch.randn(q.shape[0], hq * dv + (-hq * dv) % 8, generator=gen).to(dtype)
    extras = dict(gate=logits.cuda(), gate_offset=0, feature_gate=True) if keep else {}
    out = attend(q, cache, dv, d == dv, table, pos, seq, scale=scale, window=window, keep_first=keep, softcap=softcap or 0.0,
                 difference=(share, eps), out_scale=factor, **extras)
    at, errors = 0, []
    for i, (n, q_len) in enumerate(work):
        mask, rows = plain.seen(n, window, keep)[n - q_len:], slice(at, at + q_len)
        for h in range(hq):
            g = h * hkv // hq
            a = [plain.softmax_weights(q[rows, h, m * half:(m + 1) * half].double(), ks[i][:, g, m * half:(m + 1) * half].double(),
                                       scale, mask, softcap) @ vs[i][:, g].double() for m in (0, 1)]
            raw = a[0] - share * a[1]
            o = plain.rms(raw, eps) * factor
            if keep:
                o = o * torch.sigmoid(logits[rows, h * dv:(h + 1) * dv].double())
            err = (out[rows, h * dv:(h + 1) * dv] - o).abs().amax(-1)
            # rounded probabilities weigh more where the difference is small beside its parts: what the norm multiplies
            errors.append(err * torch.clamp((raw * raw).mean(-1).sqrt() / (vs[i].double() ** 2).mean().sqrt(), max=1.0))
        at += q_len
    worst = float(torch.cat(errors).max())
    assert worst <= (2e-5 if dtype == torch.float32 else 2.5e-2), worst


def test_differential_attention_with_many_heads_a_key():
    """Eight query heads a key head fill the sixteen rows of the decode kernel's products; more run on the general kernel."""
    from tinyinfer_b200 import ops
    gen = torch.Generator().manual_seed(1)
    for hq, hkv in ((16, 2), (5, 1), (18, 2)):
        work = [(700, 1), (40, 1), (129, 129)]
        q, cache, ks, vs, table, pos, seq = attention_case(work, 16, hq, hkv, 128, 128, torch.bfloat16, None, 0, gen)
        assert ops.attention_tensor_cores_ok(q, cache, 2) == (hq // hkv <= 8)
        out = attend(q, cache, 128, True, table, pos, seq, scale=0.125, difference=(0.5, 1e-6))
        at = 0
        for i, (n, q_len) in enumerate(work):
            mask = plain.seen(n, None)[n - q_len:]
            for h in range(hq):
                g = h * hkv // hq
                a = [plain.softmax_weights(q[at:at + q_len, h, m * 64:(m + 1) * 64].double(), ks[i][:, g, m * 64:(m + 1) * 64].double(),
                                           0.125, mask) @ vs[i][:, g].double() for m in (0, 1)]
                raw = a[0] - 0.5 * a[1]
                err = (out[at:at + q_len, h * 128:(h + 1) * 128] - plain.rms(raw, 1e-6)).abs().amax(-1)
                assert float((err * torch.clamp((raw * raw).mean(-1).sqrt(), max=1.0)).max()) <= 2.5e-2, (hq, i, h)
            at += q_len


@pytest.mark.parametrize("m", [1, 3, 16, 20, 33, 64, 65, 130, 300, 700, 2500])
@pytest.mark.parametrize("inter,k", [(56, 72), (136, 128), (376, 248), (1024, 512)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_gated_product_with_biases(m, inter, k, dtype):
    from tinyinfer_b200 import ops
    gen = torch.Generator().manual_seed(m + inter)
    x, w, b = torch.randn(m, k, generator=gen).to(dtype), (torch.randn(2 * inter, k, generator=gen) / k ** 0.5).to(dtype), torch.randn(2 * inter, generator=gen)
    got = ops.gated_linear(x.cuda(), w.cuda(), bias=b.cuda()).cpu().double()
    ops.check_kernel_status()
    z = x.double() @ w.double().t() + b.double()
    want = z[:, :inter] * torch.sigmoid(z[:, :inter]) * z[:, inter:]
    assert (got - want).abs().max() <= (5e-5 if dtype == torch.float32 else 1e-2) * want.abs().max()


@pytest.mark.parametrize("tokens", [1, 5, 64, 700, 3000])
@pytest.mark.parametrize("experts,top,hidden,ff", [(5, 3, 72, 24), (8, 1, 128, 64), (64, 6, 64, 32), (300, 2, 40, 8), (1, 1, 40, 16)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_experts_named_by_a_table(tokens, experts, top, hidden, ff, dtype):
    """Routing of three layers in one launch, the clamped activation, and the sum in the residual's own kernel."""
    from tinyinfer_b200 import ops
    gen = torch.Generator().manual_seed(tokens + experts)
    vocab = 50
    tables = torch.rand(3, vocab, experts, generator=gen).argsort(-1)[..., :top].to(torch.int32).contiguous()
    ids = torch.randint(0, vocab, (tokens,), generator=gen)
    x = torch.randn(tokens, hidden, generator=gen).to(dtype)
    tile = ops.expert_tile_rows_of(tokens, hidden, dtype, experts, top, ff)
    routes = ops.route_by_tables(ids.to(torch.int32).cuda(), tables.cuda(), experts, tile)
    assert len(routes) == 3
    for r, table in zip(routes, tables):
        chosen, slot, token_of = r.chosen.cpu().long(), r.slot_of.cpu().long(), r.token_of.cpu().long()
        assert torch.equal(chosen, table[ids].long())
        assert torch.equal(slot.flatten().sort().values, torch.arange(tokens * top))
        assert torch.equal(token_of[slot], torch.arange(tokens)[:, None].expand(-1, top))
        by_slot = torch.empty(tokens * top, dtype=torch.long)
        by_slot[slot.flatten()] = chosen.flatten()
        assert bool((by_slot[1:] >= by_slot[:-1]).all())                     # expert order
        n = int(r.num_tiles.item())
        tiles = r.tiles.cpu()[:n].tolist()
        assert sum(t[2] for t in tiles) == tokens * top and all(0 < t[2] <= tile for t in tiles)
        at = 0
        for e, first, rows in tiles:
            assert first == at and bool((by_slot[first:first + rows] == e).all())
            at += rows
    w = {f"e{e}.{n}": (torch.randn(s, generator=gen) / s[1] ** 0.5).to(dtype) for e in range(experts)
         for n, s in (("gate", (ff, hidden)), ("up", (ff, hidden)), ("down", (hidden, ff)))}
    up = torch.stack([torch.cat([w[f"e{e}.gate"], w[f"e{e}.up"]]) for e in range(experts)]).cuda()
    down = torch.stack([w[f"e{e}.down"] for e in range(experts)]).cuda()
    rows = ops.expert_linear(ops.clamped_glu(ops.expert_linear(x.cuda(), up, routes[1], up=True, activation=False), 0.6, plain.GLU_ALPHA),
                             down, routes[1], up=False)
    wd = {n: t.double() for n, t in w.items()}
    wd["table"] = tables[1]
    some = list(range(0, tokens, max(1, tokens // 40)))
    f = zh.moe(experts, top, ff, limit=0.6)
    want = plain.table_experts(wd, f, x[some].double(), ids[some].tolist())
    tol = (3e-5 if dtype == torch.float32 else 2e-2) * max(1.0, float(want.abs().max()))
    got = ops.experts_combine(rows, x.cuda(), routes[1], experts).cpu().double()
    assert (got[some] - want).abs().max() <= tol
    stream = torch.randn(tokens, hidden, generator=gen)
    y = torch.randn(tokens, hidden, generator=gen).to(dtype)
    xd = stream.cuda()
    ops.residual_step(xd, ops.ResidualUpdate(y.cuda(), factor=0.5, second=ops.ExpertRows(rows, routes[1].slot_of, 1.0 / top)),
                      torch.ones(hidden).cuda(), 1e-5, dtype)
    assert (xd.cpu().double()[some] - (stream[some].double() + 0.5 * (y[some].double() + want))).abs().max() <= tol


@pytest.mark.parametrize("width", [72, 50, 1024])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_residual_with_two_sublayers_and_its_projection(width, dtype):
    """x + (y1 + y2) and its norm; then W [x; x0], for which a bfloat16 model's x keeps sixteen bits of mantissa: an x of a few
    thousand projects to within float32-like distance, which eight bits could not."""
    from tinyinfer_b200 import ops
    gen = torch.Generator().manual_seed(width)
    n, vocab = 37, 20
    x, y1, y2 = 3000 * torch.randn(n, width, generator=gen), torch.randn(n, width, generator=gen).to(dtype), torch.randn(n, width, generator=gen).to(dtype)
    table, ids = torch.randn(vocab, width, generator=gen).to(dtype), torch.randint(0, vocab, (n,), generator=gen)
    w = 1 + 0.2 * torch.randn(width, generator=gen)
    u = x.double() + 0.5 * (y1.double() + y2.double())
    update = lambda: ops.ResidualUpdate(y1.cuda(), factor=0.5, second=y2.cuda())
    xd = x.cuda()
    rows = ops.residual_enter(xd, update(), table.cuda(), ids.to(torch.int32).cuda(), 1.0)
    assert torch.equal(xd.cpu(), x)
    parts = rows.cpu().double().reshape(n, -1, width)
    assert torch.equal(parts[:, -1], table[ids].double())
    assert parts.shape[1] == (2 if dtype == torch.float32 else 3)
    assert (parts[:, :-1].sum(1) - u).abs().max() <= 2.0 ** -16 * u.abs().max()
    bare = ops.residual_enter(xd, None, table.cuda(), ids.to(torch.int32).cuda(), 1.0).cpu().double().reshape(n, -1, width)
    assert (bare[:, :-1].sum(1) - x.double()).abs().max() <= 2.0 ** -16 * x.abs().max()
    same, h = ops.residual_step(xd, update(), w.cuda(), 1e-5, dtype)
    assert same is xd and (xd.cpu().double() - u).abs().max() <= 1e-3
    want = plain.rms(u, 1e-5) * w.double()
    assert (h.cpu().double() - want).abs().max() <= (1e-5 if dtype == torch.float32 else 8e-3) * want.abs().max()


@pytest.mark.parametrize("rows,ff", [(1, 24), (33, 20), (700, 704), (5, 8)])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_clamped_glu_in_both_forms(rows, ff, dtype):
    from tinyinfer_b200 import ops
    z = (3 * torch.randn(rows, 2 * ff, generator=torch.Generator().manual_seed(ff))).to(dtype)
    g, u = torch.clamp(z[:, :ff].double(), max=1.2), torch.clamp(z[:, ff:].double(), -1.2, 1.2)
    want = g * torch.sigmoid(1.702 * g) * (u + 1)
    got = ops.clamped_glu(z.cuda(), 1.2, 1.702).cpu().double()
    assert (got - want).abs().max() <= (1e-6 if dtype == torch.float32 else 6e-3) * want.abs().max()


# ------------------------------------------------------------------ each mechanism alone
ALONE = {
    "kept": zh.config([zh.layer("attention", zh.kept(6, 2, 20, scale=0.35, rot=12, size=9, keep=4), None)]),
    "kept_planes": zh.config([zh.layer("attention", zh.kept(4, 2, 64, scale=0.2, rot=32, size=30, keep=17), None)]),
    "difference": zh.config([zh.layer("attention_2", zh.difference(6, 2, 10, 28, scale=0.35, rot=8, size=9, softcap=2.0), None)]),
    "difference_planes": zh.config([zh.layer("attention_2", zh.difference(4, 2, 32, 64, scale=0.2, rot=32, size=30, diff=0.7,
                                                                          blend=zh.scaling(4.0, 1.0, 2.0, 60)), None)]),
    "dense": zh.config([zh.layer("attention", zh.kept(1, 1, 8, size=3), zh.dense(56))]),
    "experts": zh.config([zh.layer("attention", zh.kept(1, 1, 8, size=3), zh.moe(9, 4, 24))]),
    "looped": zh.config([zh.layer("attention", zh.kept(2, 1, 8, size=4, keep=2), None),
                         zh.layer("attention_2", zh.difference(2, 1, 8, 8, size=6), zh.moe(3, 2, 8))], loop=(0, 2, 4)),
}


@pytest.mark.parametrize("name", sorted(ALONE))
def test_one_mechanism_alone(tmp_path, name):
    cfg = ALONE[name]
    folder = zh.write_folder(tmp_path / "m", cfg, seed=11)
    requests = zh.random_requests(cfg, [75, 1, 2, 19], seed=4)
    want = zh.plain_logits(folder, requests)
    for steps in (helpers.trace_whole(requests), helpers.trace_chunked(requests, seed=3), helpers.trace_decode_tail(requests, tail=80)):
        got, _ = run(folder, "float32", steps, page=8)
        assert helpers.first_bad(got, want, TOL["float32"]) is None


@pytest.mark.parametrize("name", ["MIX", "WIDE", "ONE"])
def test_residual_after_every_layer_run(tmp_path, name):
    """The float32 stream after every layer run of a prompt (a looped layer counts each time), not only the logits."""
    from tinyinfer_b200 import ops
    from tinyinfer_b200.engine.replay import TraceSession
    cfg = getattr(zh, name)
    folder = zh.write_folder(tmp_path / "m", cfg, seed=2)
    tokens = zh.random_requests(cfg, [23], seed=1)["r0"]
    c, w = zh.read_folder(folder)
    want = []
    zh.forward(c, w, tokens, residuals=want)
    session = TraceSession(folder, "float32", 64, page_size=8, cuda_graphs=False)
    got = []
    for block in session.model.blocks:          # a block returns the stream and the update that the next norm applies
        inner = block.forward_linked

        def watched(x, link, next_norm, step, cache, _inner=inner):
            out = _inner(x, link, next_norm, step, cache)
            (stream, update), _ = out
            second = update.second
            if isinstance(second, ops.ExpertRows):
                second = second.weight * second.rows[second.slots.long()].sum(1)
            got.append((stream + update.y + (0 if second is None else second)).detach().cpu().double())
            return out
        block.forward_linked = watched
    session.run_step({"step": 0, "entries": [{"id": "a", "tokens": tokens, "want": [len(tokens) - 1]}], "end": ["a"]})
    assert len(got) == len(want) == len(plain.run_order(cfg))
    for i, rows in enumerate(got):
        assert (rows - want[i]).abs().max() <= 2e-5 * want[i].abs().max(), i


# ------------------------------------------------------------------ whole models, every cut
def traces_for(requests, max_live=4):
    return {"whole": helpers.trace_whole(requests), "tail": helpers.trace_decode_tail(requests, tail=32),
            "chunked": helpers.trace_chunked(requests, seed=1), "mixed": helpers.trace_mixed(requests, seed=2, max_live=max_live)}


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name,page", [("MIX", 8), ("WIDE", 16), ("ONE", 4)])
def test_every_cut_matches_plain(tmp_path, name, page, dtype):
    cfg = getattr(zh, name)
    folder = zh.write_folder(tmp_path / name, cfg, seed=3, dtype=dtype)
    requests = zh.random_requests(cfg, LENGTHS, seed=5)
    want = zh.plain_logits(folder, requests)
    results = {}
    for tag, steps in traces_for(requests).items():
        got, session = run(folder, dtype, steps, page, max_live=4)
        assert {r: len(v) for r, v in got.items()} == {r: len(t) for r, t in requests.items()}, tag
        assert agrees(got, want, dtype), (tag, helpers.first_bad(got, want, TOL[dtype]), np.sort(row_errors(got, want))[-8:])
        if tag == "mixed":
            stats = session.runner.manager.stats()
            assert all(g["pages_taken"] > g["pages"] for g in stats["groups"]), "pages were not used again"
        results[tag] = got
    for tag in ("tail", "chunked", "mixed"):        # the cuts against each other: rounding only
        assert agrees(results[tag], {r: np.stack([results["whole"][r][p] for p in range(len(t))]) for r, t in requests.items()},
                      dtype), tag


def test_two_live_requests_serve_many(tmp_path):
    """Pages (those a window has passed, those of kept positions, those of finished requests) go to new requests."""
    cfg = zh.MIX
    folder = zh.write_folder(tmp_path / "m", cfg, seed=8)
    requests = zh.random_requests(cfg, [30, 9, 41, 2, 17, 55, 5, 26], seed=9)
    want = zh.plain_logits(folder, requests)
    steps = helpers.trace_mixed(requests, seed=4, max_live=2, decode_tail=6)
    got, session = run(folder, "float32", steps, page=4, max_live=2)
    assert helpers.first_bad(got, want, TOL["float32"]) is None
    assert session.runner.manager.stats()["free_state_slots"] == 2


def test_batch_of_unequal_requests_equals_each_alone(tmp_path):
    cfg = zh.WIDE
    folder = zh.write_folder(tmp_path / "m", cfg, seed=5)
    requests = zh.random_requests(cfg, [50, 3, 128, 17], seed=2)
    together = [{"step": 0, "entries": [{"id": r, "tokens": t, "want": list(range(len(t)))} for r, t in requests.items()],
                 "end": list(requests)}]
    got, _ = run(folder, "float32", together, page=16)
    alone, _ = run(folder, "float32", helpers.trace_whole(requests), page=16)
    want = zh.plain_logits(folder, requests)
    assert helpers.first_bad(got, want, TOL["float32"]) is None
    scale = max(float(np.abs(w).max()) for w in want.values())
    assert max(float(np.abs(got[r][p] - alone[r][p]).max()) for r in requests for p in got[r]) / scale <= 1e-5


def test_a_request_left_out_of_steps_goes_on(tmp_path):
    """A request pauses for some steps while others run and end (their pages change hands meanwhile)."""
    cfg = zh.MIX
    folder = zh.write_folder(tmp_path / "m", cfg, seed=4)
    requests = zh.random_requests(cfg, [40, 21, 33], seed=7)
    a, b, c = (requests[f"r{i}"] for i in range(3))
    want = zh.plain_logits(folder, requests)
    every = lambda toks, lo, hi: {"tokens": toks[lo:hi], "want": list(range(hi - lo))}
    steps = [
        {"step": 0, "entries": [dict(id="r0", **every(a, 0, 13)), dict(id="r1", **every(b, 0, 21))], "end": ["r1"]},
        {"step": 1, "entries": [dict(id="r2", **every(c, 0, 2))], "end": []},
        {"step": 2, "entries": [dict(id="r2", **every(c, 2, 33))], "end": ["r2"]},
        {"step": 3, "entries": [dict(id="r0", **every(a, 13, 14))], "end": []},
        {"step": 4, "entries": [dict(id="r0", **every(a, 14, 40))], "end": ["r0"]},
    ]
    got, _ = run(folder, "float32", steps, page=8, max_live=2)
    assert helpers.first_bad(got, want, TOL["float32"]) is None


# ------------------------------------------------------------------ edges of windows and kept positions, far keys, first tokens
def edge_config(kind, size, keep, planes):
    if kind == "attention":
        d = 64 if planes else 12
        m = zh.kept(4, 2, d, scale=4.0 / d ** 0.5, rot=d // 4 * 2, size=size, keep=keep)
    else:
        d, dv = (32, 64) if planes else (12, 20)
        m = zh.difference(4, 2, d, dv, scale=3.0 / d ** 0.5, rot=d // 4 * 2, size=size, diff=0.4)
    return zh.config([zh.layer(kind, m, None)], width=64)


@pytest.mark.parametrize("dtype,planes", [("float32", False), ("float32", True), ("bfloat16", True)])
@pytest.mark.parametrize("kind,size,keep", [("attention", 24, 3), ("attention", 37, 16), ("attention", 20, 17), ("attention_2", 24, 0),
                                            ("attention_2", 37, 0)])
def test_keys_just_inside_and_outside(tmp_path, kind, size, keep, planes, dtype):
    """One token is replaced. At the positions that may see it the logits move and agree with the plain statement; at the
    first position that may not, and at all behind it, they are what they were; a kept token is seen to the end. In prompts and
    token by token, for tokens at the edges of windows, of the kept positions and of pages."""
    cfg = edge_config(kind, size, keep, planes)
    folder = zh.write_folder(tmp_path / "m", cfg, seed=31, dtype=dtype)
    base = zh.random_requests(cfg, [4 * size + 5], seed=3)["r0"]
    n = len(base)
    places = sorted({0, max(0, keep - 1), keep, keep + 1, size - 1, size, 2 * size - 1, 15, 16, 47, 48, 2 * size + 3} - {n})
    requests = {"base": base}
    for p in places:
        requests[f"p{p}"] = base[:p] + [(base[p] + 1) % cfg["vocab"]] + base[p + 1:]
    want = zh.plain_logits(folder, requests)
    scale = np.abs(want["base"]).max()
    for steps in (helpers.trace_whole(requests), helpers.trace_decode_tail(requests, tail=3 * size), helpers.trace_chunked(requests, seed=5)):
        got, _ = run(folder, dtype, steps, page=16)
        assert agrees(got, want, dtype)
        for p in places:
            last = n - 1 if p < keep else p + size - 1        # the last position that sees p
            moved = [float(np.abs(got[f"p{p}"][i] - got["base"][i]).max()) / scale for i in range(n)]
            should = [float(np.abs(want[f"p{p}"][i] - want["base"][i]).max()) / scale for i in range(n)]
            assert max(moved[:p], default=0.0) <= 1e-6 and max(moved[last + 1:], default=0.0) <= 1e-6, p
            assert max(should[last + 1:], default=0.0) == 0.0
            if last < n and should[last] > 10 * TOL[dtype]:
                assert moved[last] > 5 * TOL[dtype], p
    # the premise: for some of these places the very last position that sees the token moves by far more than the tolerance
    seen = 0
    for p in places:
        last = n - 1 if p < keep else p + size - 1
        seen += last < n and np.abs(want[f"p{p}"][last] - want["base"][last]).max() / scale > 10 * TOL["float32"]
    assert seen >= 3


def far_config():
    """Windows that reach far back, kept positions, and scores sharp enough that one key takes nearly all of a head."""
    return zh.config([
        zh.layer("attention", zh.kept(4, 2, 16, scale=2.0, rot=8, size=300, keep=40), zh.dense(48)),
        zh.layer("attention_2", zh.difference(4, 2, 16, 24, scale=2.0, rot=8, size=640, softcap=25.0,
                                              blend=zh.scaling(4.0, 1.0, 4.0, 256)), zh.moe(5, 2, 24)),
    ], width=64, loop=(0, 2, 2))


def test_far_tokens_carry_the_result(tmp_path):
    """Positions around the borders of pages and of the kernels' key tiles are decoded one by one; replacing the first 64
    tokens moves the last logits by far more than the tolerance, so a missing or misplaced row shows."""
    cfg = far_config()
    folder = zh.write_folder(tmp_path / "m", cfg, seed=21)
    requests = zh.random_requests(cfg, [700], seed=13)
    tokens = requests["r0"]
    want = zh.plain_logits(folder, requests)
    c, w = zh.read_folder(folder)
    other = [(t + 1) % cfg["vocab"] for t in tokens[:64]] + tokens[64:]
    assert np.abs(zh.forward(c, w, other)[-60:] - want["r0"][-60:]).max() > 100 * TOL["float32"] * np.abs(want["r0"]).max()
    for steps in (helpers.trace_whole(requests), helpers.trace_decode_tail(requests, tail=140), helpers.trace_chunked(requests, seed=7)):
        got, _ = run(folder, "float32", steps, page=16)
        assert helpers.first_bad(got, want, 2 * TOL["float32"]) is None
    folder16 = zh.write_folder(tmp_path / "m16", cfg, seed=21, dtype="bfloat16")
    want16 = zh.plain_logits(folder16, requests)
    for steps in (helpers.trace_whole(requests), helpers.trace_decode_tail(requests, tail=140), helpers.trace_chunked(requests, seed=7)):
        got, _ = run(folder16, "bfloat16", steps, page=16)
        err = row_errors(got, want16)
        assert np.isfinite(err).all() and np.median(err) <= 4e-2 and (err > 0.25).mean() <= 0.03, np.sort(err)[-5:]


@pytest.mark.parametrize("dtype,dims", [("float32", (16, 16)), ("bfloat16", (64, 64))])
@pytest.mark.parametrize("kind", ["attention", "attention_2"])
def test_one_far_key_among_hundreds(tmp_path, kind, dtype, dims):
    """Scores are scaled so that one early key outscores all others by a wide margin: the logits at the end hang on that
    token's value. Replacing the token changes them; the engine agrees with the plain statement on both, decoded through the
    cache, at several page sizes. In the windowed mixer the far token is a kept one, hundreds of positions behind the window."""
    d, dv = dims
    if kind == "attention":
        m = zh.kept(2, 1, d, scale=8.0 / d ** 0.5, size=50, keep=101)
    else:
        m = zh.difference(2, 1, dv // 2, dv, scale=8.0 / (dv // 2) ** 0.5, size=400, diff=0.3)
    cfg = zh.config([zh.layer(kind, m, None)], width=32)
    folder = zh.write_folder(tmp_path / "m", cfg, seed=5, dtype=dtype)
    base = zh.random_requests(cfg, [300], seed=3)["r0"]
    c, w = zh.read_folder(folder)
    full = zh.forward(c, w, base)
    moves = {}
    for p in (3, 15, 16, 17, 31, 32, 63, 64, 65, 100):
        other = list(base)
        other[p] = (other[p] + 1) % cfg["vocab"]
        moves[p] = float(np.abs(zh.forward(c, w, other)[-40:] - full[-40:]).max())
    far = max(moves, key=moves.get)
    assert moves[far] > (1e-2 if dtype == "float32" else 0.15) * np.abs(full).max()
    changed = list(base)
    changed[far] = (changed[far] + 1) % cfg["vocab"]
    requests = {"r0": base, "r1": changed}
    want = zh.plain_logits(folder, requests)
    for page in ((4, 16, 64) if dtype == "float32" else (16, 64)):
        got, _ = run(folder, dtype, helpers.trace_decode_tail(requests, tail=40), page=page)
        assert agrees(got, want, dtype), page


def test_the_first_tokens(tmp_path):
    """Position zero (no angle, a softmax of one key), then the next few, kept ones and others, as prompts of one to twelve
    tokens and decoded one by one from the start."""
    cfg = zh.MIX
    folder = zh.write_folder(tmp_path / "m", cfg, seed=12)
    requests = zh.random_requests(cfg, [1, 2, 3, 4, 5, 6, 9, 10, 11, 12], seed=8)
    want = zh.plain_logits(folder, requests)
    for steps in (helpers.trace_whole(requests), helpers.trace_decode_tail(requests, tail=12)):
        got, _ = run(folder, "float32", steps, page=4)
        assert helpers.first_bad(got, want, TOL["float32"]) is None


# ------------------------------------------------------------------ long decoding through graphs
@pytest.mark.parametrize("name", ["MIX", "WIDE"])
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_replays_graphs(tmp_path, dtype, name):
    """The tables route a step's own tokens in a replayed graph too; windows pass over many decoded tokens."""
    cfg = getattr(zh, name)
    folder = zh.write_folder(tmp_path / "m", cfg, seed=6, dtype=dtype)
    requests = zh.random_requests(cfg, [160, 150, 155], seed=1)
    want = zh.plain_logits(folder, requests)
    steps = [{"step": 0, "entries": [{"id": r, "tokens": t[:4], "want": [0, 1, 2, 3]} for r, t in requests.items()], "end": []}]
    for p in range(4, 150):
        steps.append({"step": p, "entries": [{"id": r, "tokens": [t[p]], "want": [0]} for r, t in requests.items()],
                      "end": list(requests) if p == 149 else []})
    got, session = run(folder, dtype, steps, page=16)
    assert session.runner.graph_replays > 100
    assert agrees(got, {r: w[:150] for r, w in want.items()}, dtype)


# ------------------------------------------------------------------ generation through the entry point
@pytest.mark.parametrize("dtype,tol", [("float32", 1e-4), ("bfloat16", 8e-2)])
def test_greedy_generation_through_the_scheduler(tmp_path, dtype, tol):
    from tinyinfer_b200 import LLM
    from tinyinfer_b200.sampling import SamplingParams
    cfg = zh.MIX
    folder = zh.write_folder(tmp_path / "m", cfg, seed=3, dtype=dtype)
    llm = LLM(folder, dtype=dtype, max_num_batched_tokens=24, max_num_seqs=3, kvcache_block_size=8,
              num_kvcache_blocks=40, prefill_chunk=9, max_model_len=128)
    assert llm.config.enable_prefix_caching is False          # a window gives pages back
    prompts = list(zh.random_requests(cfg, [1, 7, 16, 33, 50], seed=6).values())
    outs = llm.generate(prompts, SamplingParams(greedy=True, max_tokens=10))
    c, w = zh.read_folder(folder)
    for p, o in zip(prompts, outs):
        assert o["all_token_ids"] == p + o["token_ids"] and len(o["token_ids"]) == 10
        logits = zh.forward(c, w, p + o["token_ids"])
        for i, tok in enumerate(o["token_ids"]):          # teacher forcing: the token has (nearly) the largest plain logit
            row = logits[len(p) - 1 + i]
            assert row.max() - row[tok] <= tol * np.abs(logits).max()
    assert not llm.runner.manager.live_requests
    llm.runner.manager.check_consistency()
    llm.close()


def test_command_line_generates_with_a_folder_and_with_a_preset(tmp_path):
    import json
    import subprocess
    import sys
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    folder = zh.write_folder(tmp_path / "m", zh.ONE, seed=3)
    common = ["--dtype", "fp32", "--prompt-ids", "5,17,3,200", "--prompt-len", "9", "--greedy", "--max-tokens", "6",
              "--max-num-seqs", "2", "--max-num-batched-tokens", "16", "--block-size", "4", "--num-kvcache-blocks", "32",
              "--max-model-len", "64"]
    res = subprocess.run([sys.executable, str(root / "examples" / "generate.py"), "--model", str(folder)] + common,
                         capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]
    rows = [json.loads(l) for l in res.stdout.splitlines() if l.startswith("{")]
    assert len(rows) == 2 and all(len(r["token_ids"]) == 6 for r in rows)
    c, w = zh.read_folder(folder)
    logits = zh.forward(c, w, [5, 17, 3, 200] + rows[0]["token_ids"])
    for i, tok in enumerate(rows[0]["token_ids"]):
        assert logits[3 + i].max() - logits[3 + i][tok] <= 1e-4 * np.abs(logits).max()
    res = subprocess.run([sys.executable, str(root / "examples" / "generate.py"), "--random-config", "zetonex-tiny"] + common,
                         capture_output=True, text=True, timeout=600)
    assert res.returncode == 0, res.stderr[-2000:]


def test_trace_runner_program(tmp_path):
    """The replay program itself: steps on standard input, a file of logits per step that wants some, 'done' lines."""
    import json
    import subprocess
    from pathlib import Path
    root = Path(__file__).resolve().parent.parent
    cfg = zh.ONE
    folder = zh.write_folder(tmp_path / "m", cfg, seed=9, dtype="bfloat16")
    requests = zh.random_requests(cfg, [20, 70, 9], seed=2)
    steps = helpers.trace_mixed(requests, seed=1, max_live=3, decode_tail=5)
    out = tmp_path / "out"
    out.mkdir()
    res = subprocess.run([str(root / "bin" / "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out),
                          "--max-tokens", str(helpers.peak_tokens(steps))], input="".join(json.dumps(s) + "\n" for s in steps),
                         capture_output=True, text=True, timeout=1200)
    assert res.returncode == 0, res.stderr[-2000:]
    assert [l for l in res.stdout.splitlines() if l.startswith("done ")] == [f"done {s['step']}" for s in steps]
    want = zh.plain_logits(folder, requests)
    upto = {}
    for s in steps:
        wanted = [(e["id"], upto.get(e["id"], 0) + p) for e in s["entries"] for p in e["want"]]
        for e in s["entries"]:
            upto[e["id"]] = upto.get(e["id"], 0) + len(e["tokens"])
        rows = np.fromfile(out / f"{s['step']}.f32", dtype="<f4").reshape(len(wanted), cfg["vocab"])
        for row, (rid, p) in zip(rows, wanted):
            assert np.abs(row - want[rid][p]).max() <= TOL["float32"] * np.abs(want[rid]).max()


def random_config(seed):
    """A model of random sizes and layer order: odd head counts and sizes, partial and no rotation, with and without
    frequency scaling and cap, windows from one key on or none, kept positions or none, with and without feed-forward, loops
    anywhere or none."""
    rng = random.Random(seed)
    layers = []
    for _ in range(rng.randint(2, 6)):
        roll = rng.random()
        mlp = None if roll < 0.2 else zh.dense(rng.choice([24, 56, 136]))
        if roll > 0.5:
            experts = rng.randint(1, 12)
            mlp = zh.moe(experts, rng.randint(1, min(6, experts)), rng.choice([8, 24, 40]), limit=rng.choice([0.5, 1.0, 7.0]))
        kv, size = rng.randint(1, 3), rng.choice([None, 1, 2, 5, 16, 33, 64, 200])
        heads, base = kv * rng.randint(1, 3), rng.choice([100.0, 10000.0, 1e6])
        if rng.random() < 0.5:
            d = rng.choice([8, 12, 20, 40, 64])
            m = zh.kept(heads, kv, d, scale=rng.uniform(0.1, 0.5), rot=rng.choice([0, 4, d // 4 * 2, d]), base=base, size=size,
                        keep=rng.choice([0, 1, 4, 17, 90]) if size else 0)
            layers.append(zh.layer("attention", m, mlp))
        else:
            d = rng.choice([4, 6, 20, 32, 64])
            m = zh.difference(heads, kv, d, 2 * d if rng.random() < 0.5 else rng.choice([8, 24, 36]), scale=rng.uniform(0.1, 0.5),
                              rot=rng.choice([0, 4, d // 4 * 2, d // 2 * 2]), base=base, size=size, diff=rng.choice([0.0, 0.25, 0.8]),
                              softcap=rng.choice([None, 2.0, 30.0]), blend=rng.choice([None, zh.scaling(8.0, 1.0, 4.0, 64)]))
            layers.append(zh.layer("attention_2", m, mlp))
    n = len(layers)
    start = rng.randrange(n)
    loop = None if rng.random() < 0.3 else (start, rng.randint(start + 1, n), rng.randint(1, 3))
    return zh.config(layers, vocab=rng.choice([97, 256, 300]), width=rng.choice([40, 72, 100, 136]), eps=rng.choice([1e-5, 1e-6]),
                     logit_scale=rng.choice([1.0, 0.3, 2.5]), loop=loop)


@pytest.mark.parametrize("seed", [1, 2, 3, 4, 5, 6, 7, 8])
def test_models_of_random_sizes_and_orders(tmp_path, seed):
    cfg = random_config(seed)
    page = [4, 8, 16, 32, 64, 16, 16, 8][seed - 1]
    requests = zh.random_requests(cfg, [70, 1, 37, 150, 2, 64], seed=seed)
    folder = zh.write_folder(tmp_path / "m", cfg, seed=seed)
    want = zh.plain_logits(folder, requests)
    for steps in (helpers.trace_whole(requests), helpers.trace_mixed(requests, seed=seed, max_live=3, decode_tail=20)):
        got, _ = run(folder, "float32", steps, page, max_live=3)
        assert helpers.first_bad(got, want, TOL["float32"]) is None, cfg
    folder16 = zh.write_folder(tmp_path / "m16", cfg, seed=seed, dtype="bfloat16")
    got, _ = run(folder16, "bfloat16", helpers.trace_mixed(requests, seed=seed, max_live=3, decode_tail=20), page, max_live=3)
    err = row_errors(got, zh.plain_logits(folder16, requests))
    assert np.isfinite(err).all() and np.median(err) <= TOL["bfloat16"] / 2, (np.median(err), cfg)
