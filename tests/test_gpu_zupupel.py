"""Zupupel stacks on a GPU: every kernel against a plain statement, the engine's schedules against each other and against the
float64 model, captured decode windows, and the trace program."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import composed_driver as D  # noqa: E402
import oracle_zupupel as O  # noqa: E402
from oracle_composed import distance, distances, tokens  # noqa: E402

pytestmark = pytest.mark.gpu
F64 = torch.float64
BF = torch.bfloat16
BOTH = pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])


@pytest.fixture(autouse=True)
def _inference():
    with torch.no_grad():
        yield


def _rand(seed, *s, dtype=torch.float32):
    return torch.randn(*s, device="cuda", generator=torch.Generator(device="cuda").manual_seed(seed)).to(dtype)


def _i32(v):
    return torch.tensor(v, dtype=torch.int32, device="cuda")


def _tol(dtype):
    return 1e-2 if dtype == BF else 1e-5


def _close(got, want, tol):
    err = (got.to(F64).cpu() - want.to(F64).cpu()).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), (err, want.abs().max().item())


def _ok():
    from relax_b200.ops import cuda as C

    torch.cuda.synchronize()
    C.check_error_flag()


# ---------------------------------------------------------------------------------------------------- around attention


@BOTH
@pytest.mark.parametrize("H,G,dim,vdim,rot,halves", [(8, 2, 128, 128, 64, True), (6, 2, 18, 13, 10, True), (5, 5, 7, 9, 4, False), (3, 1, 144, 200, 144, True),
                                                     (4, 1, 64, 24, 0, True), (4, 2, 40, 48, 16, False), (4, 2, 40, 48, 24, True), (40, 4, 128, 64, 128, True)])
def test_projection_inputs(dtype, H, G, dim, vdim, rot, halves):
    from relax_b200 import ops
    from relax_b200.rollout.composed import head_pitch

    T, eps, dp, vp = 9, 1e-2, head_pitch(dim), head_pitch(vdim)
    x = _rand(1, T, (H * dim + G * (dim + vdim) + 71) // 8 * 8, dtype=dtype)
    x[:, :dim] *= 6
    qw, kw = 1 + _rand(2, H * dim, dtype=dtype), 1 + _rand(3, G * dim, dtype=dtype)
    pos = [0, 1, 2, 63, 64, 1000, 5000, 40000, 100000]
    table = ops.rope_table(_i32(pos) + 1, -1, torch.tensor([3e4 ** (-2 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F64, device="cuda")) if rot else None
    kp, vp_ = (torch.full((40, G, n), 7.0, dtype=dtype, device="cuda") for n in (dp, vp))
    slots = torch.tensor([3, 39, 0, 17, 16, 15, 31, 32, 8], device="cuda")
    turn = O.turn_halves if halves else O.turn_neighbours
    for w, e in (((qw, kw), eps), ((None, None), eps), ((None, None), 0.0)):
        q = ops.projection_inputs(x, *w, table, H, G, dim, vdim, dp, rot, halves, e, kp, vp_, slots)
        for got, a, n, nw in ((q, 0, H, w[0]), (kp[slots], H * dim, G, w[1])):
            want = x[:, a:a + n * dim].to(F64).cpu()
            if e:
                want = O.rms(want, 1.0 if nw is None else nw.to(F64).cpu(), eps)
            _close(got[..., :dim], turn(want.view(T, n, dim), pos, rot, 3e4), 5e-3 if dtype == BF else 3e-6)
            assert not got[..., dim:].any()
        assert torch.equal(ops.projection_inputs(x, w[0], None, table, H, G, dim, vdim, dp, rot, halves, e, None, None, slots), q)
    assert torch.equal(vp_[slots, :, :vdim], x[:, (H + G) * dim:(H + G) * dim + G * vdim].view(T, G, vdim)) and not vp_[slots, :, vdim:].any()
    other = torch.ones(40, dtype=torch.bool)
    other[slots.cpu()] = False
    assert bool((kp[other.cuda()] == 7).all()) and bool((vp_[other.cuda()] == 7).all())
    _ok()


def _tables(ctx, page, seed):
    nb = [(L + page - 1) // page for L in ctx]
    perm = torch.randperm(sum(nb) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    bt = torch.zeros(len(nb), max(nb) + 2, dtype=torch.int32)
    for s, n in enumerate(nb):
        bt[s, :n] = torch.tensor([perm.pop() for _ in range(n)])
    rows = [torch.tensor([int(bt[s, p // page]) * page + p % page for p in range(L)], device="cuda") for s, L in enumerate(ctx)]
    return bt.cuda(), rows, (sum(nb) + 3) * page


def _paged(ctx, G, dim, vdim, page, dtype, seed):
    from relax_b200.rollout.composed import head_pitch

    bt, rows, n = _tables(ctx, page, seed)
    k, v = _rand(seed, n, G, head_pitch(dim), dtype=dtype), _rand(seed + 1, n, G, head_pitch(vdim), dtype=dtype)
    k[..., dim:], v[..., vdim:] = 0, 0
    return k, v, bt, rows


def _batch(lens, ctx, bt, H, G):
    """Segments of several rows first, as the engine orders them."""
    from relax_b200.models.config import LayerSpec
    from relax_b200.rollout.composed import SegmentBatch, query_blocks, tile_tokens

    if all(n == 1 for n in lens):
        return SegmentBatch(None, None, _i32(ctx), bt, None, max_ctx_one=max(ctx))
    m = sum(1 for n in lens if n > 1)
    t = tile_tokens(LayerSpec("attention", heads=H, dim=8, vdim=8, kv_heads=G))
    cu = [sum(lens[:i]) for i in range(len(lens) + 1)]
    return SegmentBatch(None, None, _i32(ctx), bt, None, cu=_i32(cu), multi_segs=m, multi_rows=cu[m], max_ctx_one=max(ctx[m:], default=0),
                        seg_of=_i32([s for s, n in enumerate(lens) for _ in range(n)]), blocks={t: _i32(query_blocks(lens[:m], ctx, t))},
                        pos=_i32([c - n + k for n, c in zip(lens, ctx) for k in range(n)]))


def _attend(q, k, v, rows, lens, ctx, scale, window=None):
    """The plain statement, whole segments at a time."""
    out, at = [], 0
    rep = q.shape[1] // k.shape[1]
    for s, (n, L) in enumerate(zip(lens, ctx)):
        ks, vs = k[rows[s]].to(F64).repeat_interleave(rep, 1), v[rows[s]].to(F64).repeat_interleave(rep, 1)
        z = torch.einsum("thd,lhd->thl", q[at:at + n].to(F64), ks) * scale
        ahead = torch.arange(n, device="cuda")[:, None] + L - n - torch.arange(L, device="cuda")[None]
        hidden = ahead < 0 if window is None else (ahead < 0) | (ahead >= window)
        out.append(torch.einsum("thl,lhd->thd", torch.softmax(z.masked_fill(hidden[:, None], float("-inf")), -1), vs))
        at += n
    return torch.cat(out)


def test_the_vectorised_statement_equals_the_plain_one():
    k, v, bt, rows = _paged([9, 5], 2, 10, 6, 16, torch.float32, 1)
    q = _rand(3, 5, 4, 64)
    for window in (None, 1, 3, 6, 20):
        got, at = _attend(q, k, v, rows, [2, 3], [9, 5], 0.7, window), 0
        for s, (n, L) in enumerate(((2, 9), (3, 5))):
            _close(got[at:at + n], O.attend(q[at:at + n].to(F64).cpu(), k[rows[s]].to(F64).cpu(), v[rows[s]].to(F64).cpu(), L - n, 0.7, window), 1e-12)
            at += n


SHAPES = [(8, 2, 128, 128, 64), (8, 8, 64, 64, 16), (32, 4, 128, 128, 64), (16, 1, 64, 128, 32), (6, 2, 40, 24, 128), (9, 3, 128, 50, 16), (40, 2, 64, 64, 64),
          (3, 1, 144, 136, 64), (4, 2, 20, 100, 24)]


@BOTH
@pytest.mark.parametrize("H,G,dim,vdim,page", SHAPES)
@pytest.mark.parametrize("lens", [[1, 1, 1, 1, 1], [7, 2, 60, 130, 300, 1, 1], [2, 2]])
def test_windowed_paged_attention_with_a_gate(dtype, H, G, dim, vdim, page, lens):
    from relax_b200 import ops

    ctx = {5: [1, 128, 129, 1100, 16], 7: [7, 129, 700, 257, 300, 1, 650], 2: [2, 66]}[len(lens)]
    k, v, bt, rows = _paged(ctx, G, dim, vdim, page, dtype, H + dim)
    T, vo = sum(lens), (vdim + 7) // 8 * 8
    q, wide = _rand(5, T, H, k.shape[2], dtype=dtype), _rand(6, T, 16 + H * vo + 8, dtype=dtype)
    q[..., dim:] = 0
    gate = wide[:, 16:16 + H * vo]
    opened = torch.sigmoid(gate.to(F64)).view(T, H, vo)
    for window in (1, 33, 64, 130, 640, 5000):
        got = ops.paged_attention(q, k, v, _batch(lens, ctx, bt, H, G), page, 1.5 / dim ** 0.5, None, vo, window, gate).view(T, H, vo)
        want = _attend(q, k, v, rows, lens, ctx, 1.5 / dim ** 0.5, window)
        _close(got[..., :vdim], want[..., :vdim] * opened[..., :vdim], _tol(dtype))
        assert not got[..., vdim:].any()
    _ok()


@BOTH
@pytest.mark.parametrize("n", [1, 2, 40])
@pytest.mark.parametrize("window", [96, 128, 200, 1500])
def test_keys_inside_and_outside_a_window(dtype, n, window):
    """One key stands out for every row: just inside and just outside the window of the first and of the last row, around page and
    tile borders near the window's edge, the newest key and the one behind it."""
    from relax_b200 import ops

    H, G, dim, page, L = 4, 2, 128, 64, 2000
    edge = L - window
    k, v, bt, rows = _paged([L], G, dim, dim, page, dtype, 1)
    k.mul_(0.1)
    q = _rand(2, n, H, dim, dtype=dtype)
    q[:] = q[:1, :1]
    clean = k.clone()
    for where in sorted({0, edge - n - 1, edge - n, edge - n + 1, edge - 1, edge, edge + 1, edge // 64 * 64 - 1, edge // 64 * 64, L - n - 1, L - n, L - 1}):
        k.copy_(clean)
        k[rows[0][where]] = (q[0, :1] * 0.3).to(dtype)
        got = ops.paged_attention(q, k, v, _batch([n], [L], bt, H, G), page, 1.0, None, dim, window).view(n, H, dim)
        _close(got, _attend(q, k, v, rows, [n], [L], 1.0, window), _tol(dtype))
        for i in range(n):
            last = L - n + i
            near = (got[i, 0].float() - v[rows[0][where], 0].float()).abs().max() < 0.1
            assert bool(near) == (last - window < where <= last), (where, i)
    _ok()


# ---------------------------------------------------------------------------------------------------- latent rows


LATENT = [(4, 20, 6, 16), (16, 128, 32, 64), (32, 512, 64, 64), (40, 320, 48, 16), (70, 64, 64, 32), (3, 192, 100, 128), (8, 576, 64, 64), (24, 448, 128, 64)]


@BOTH
@pytest.mark.parametrize("H,rank,rot,page", LATENT)
@pytest.mark.parametrize("lens", [[1, 1, 1, 1, 1], [7, 2, 60, 130, 1]])
def test_latent_attention_with_a_rotated_part(dtype, H, rank, rot, page, lens):
    from relax_b200 import ops
    from relax_b200.rollout.composed import SegmentBatch, attention_items

    Rp, R = (rank + 63) // 64 * 64, (rank + 63) // 64 * 64 + (rot + 63) // 64 * 64
    ctx = [1, 128, 129, 1000, 16] if set(lens) == {1} else [7, 129, 700, 257, 300]
    bt, rows, total = _tables(ctx, page, H)
    pool, q = _rand(1, total, R, dtype=dtype), _rand(2, sum(lens), H, R, dtype=dtype)
    pool[:, rank:Rp], pool[:, Rp + rot:] = 0, 0
    if set(lens) == {1}:
        b = SegmentBatch(None, None, _i32(ctx), bt, None, max_ctx=max(ctx))
    else:
        width = ops.latent_columns(R, Rp)
        b = SegmentBatch(None, None, _i32(ctx), bt, None, cu=_i32([0]), max_ctx=max(ctx), items={H: _i32(attention_items(lens, ctx, H, width))},
                         item_width={H: width}, row_seg=_i32([s for s, n in enumerate(lens) for _ in range(n)]),
                         row_pos=_i32([c - n + k for n, c in zip(lens, ctx) for k in range(n)]))
    got = ops.latent_attention(q, pool, b, page, 1.5 / R ** 0.5, None, Rp)
    _close(got, _attend(q, pool[:, None], pool[:, None, :Rp], rows, lens, ctx, 1.5 / R ** 0.5), _tol(dtype))
    _ok()


@BOTH
@pytest.mark.parametrize("T", [1, 9, 150])
@pytest.mark.parametrize("H,d,r,rank,vdim", [(3, 10, 6, 20, 7), (16, 128, 64, 512, 128), (1, 8, 2, 64, 5), (5, 33, 32, 100, 40)])
def test_latent_rows_and_folded_maps(dtype, T, H, d, r, rank, vdim):
    """What a layer does around the attention: norm and rotation into the pages, queries that meet the rows, values and their gate."""
    from relax_b200 import ops

    dk, Rp, rp, vp = (d + r + 7) // 8 * 8, (rank + 63) // 64 * 64, (r + 7) // 8 * 8, (vdim + 7) // 8 * 8
    R, eps = Rp + (r + 63) // 64 * 64, 1e-3
    x = _rand(1, T, H * dk + Rp + rp + H * vp, dtype=dtype)
    raw = x.clone()
    q, c, k_rot, gate = x.split([H * dk, Rp, rp, H * vp], 1)
    q = q.view(T, H, dk)
    q[..., d + r:] = 0
    w = 1 + _rand(2, Rp, dtype=dtype)
    pos = [(37 * i) % 1000 + 100 * i for i in range(T)]
    table = ops.rope_table(_i32(pos), 0, torch.tensor([2e3 ** (-2 * i / r) for i in range(r // 2)], dtype=F64, device="cuda"))
    pool, slots = torch.full((T + 5, R), 7.0, dtype=dtype, device="cuda"), torch.randperm(T + 5, generator=torch.Generator().manual_seed(3))[:T].cuda()
    ops.latent_write(c, w, rank, eps, pool, slots, (q, k_rot, table, Rp, r, d))
    raw = raw.to(F64).cpu()
    wq = raw[:, : H * dk].view(T, H, dk)
    wq = torch.cat([wq[..., :d], O.turn_neighbours(wq[..., d:d + r], pos, r, 2e3)], -1)
    wk = O.turn_neighbours(raw[:, None, H * dk + Rp: H * dk + Rp + r], pos, r, 2e3)[:, 0]
    tol = 5e-3 if dtype == BF else 3e-6
    _close(q[..., : d + r], wq, tol)
    _close(pool[slots, :rank], O.rms(raw[:, H * dk: H * dk + rank], w[:rank].to(F64).cpu(), eps), tol)
    _close(pool[slots, Rp:Rp + r], wk, tol)
    assert not pool[slots, rank:Rp].any() and not pool[slots, Rp + r:].any() and int((pool == 7).all(1).sum()) == 5
    uk, uv = torch.zeros(H, dk, R, dtype=dtype, device="cuda"), torch.zeros(H, vp, Rp, dtype=dtype, device="cuda")
    uk[:, :d, :rank], uv[:, :vdim, :rank] = _rand(4, H, d, rank, dtype=dtype), _rand(5, H, vdim, rank, dtype=dtype) / rank ** 0.5
    i = torch.arange(r, device="cuda")
    uk[:, d + i, Rp + i] = 1.0
    ql = ops.head_linear(q, uk, False)
    _close(ql, torch.einsum("tha,hab->thb", q.to(F64), uk.to(F64)), 1e-2 if dtype == BF else 1e-5)
    assert torch.equal(ql[..., Rp:Rp + r], q[..., d:d + r])              # the rotated part passes exactly
    o = _rand(6, T, H, Rp, dtype=dtype)
    want = torch.einsum("tha,hba->thb", o.to(F64), uv.to(F64))
    _close(ops.head_linear(o, uv, True), want, 1e-2 if dtype == BF else 1e-5)
    _close(ops.head_linear(o, uv, True, gate), want * torch.sigmoid(gate.to(F64)).view(T, H, vp), 1e-2 if dtype == BF else 1e-5)
    _ok()


# ---------------------------------------------------------------------------------------------------- experts


def _moe(E, I, top, ff, groups=1, keep=1, limit=1.0):
    from relax_b200.models.config import MoESpec

    return MoESpec(experts=E, top=top, ff=ff, groups=groups, keep=keep, act="clamped_swish", limit=limit, renormalize=True, score="softmax", correction=True,
                   identity=I, group_best=1)


@pytest.mark.parametrize("T", [1, 37, 700])
@pytest.mark.parametrize("E,I,top,groups,keep", [(13, 2, 4, 5, 3), (128, 16, 8, 8, 4), (4, 2, 1, 6, 1), (3, 6, 2, 1, 1), (280, 20, 40, 3, 2), (8, 0, 8, 4, 4)])
def test_router_and_layout(T, E, I, top, groups, keep):
    from relax_b200 import ops

    N = E + I
    z, corr = _rand(E, T, N + 5) * 2, _rand(9, N, dtype=BF) * 0.2 - 0.5
    for dtype, tile in ((BF, 128), (torch.float32, 64)):
        p = ops.moe_route(z, _moe(E, I, top, 8, groups, keep), dtype, None, corr.to(dtype))
        ex, place, w, off = p.expert.cpu(), p.place.cpu(), p.weight.cpu(), p.offset.cpu()
        for t in range(0, T, max(1, T // 40)):
            s = O.weigh(z[t, :N].to(F64).cpu())
            chosen, gap = O.choose((s + corr.to(F64).cpu()).tolist(), top, groups, keep)
            if gap > 1e-6:
                assert sorted(ex[t].tolist()) == sorted(chosen)
                total = sum(s[e] for e in chosen)
                assert all(abs(w[t, j] - s[int(ex[t, j])] / total) < 1e-5 for j in range(top))
        real = ex < E
        count = torch.bincount(ex[real], minlength=E)
        assert off.tolist() == [0] + torch.cumsum(count, 0).tolist()
        flat = (off[ex.clamp(max=E - 1).long()] + place)[real]
        assert sorted(flat.tolist()) == list(range(int(real.sum())))
        tok = p.row_token.cpu()
        assert all(int(tok[ex[t, j], place[t, j]]) == t for t in range(0, T, max(1, T // 50)) for j in range(top) if real[t, j])
        want = [[e, int(off[e]) + i * tile, min(tile, int(count[e]) - i * tile), i] for e in range(E) for i in range(-(-int(count[e]) // tile))]
        assert p.tiles[: int(p.n_tiles)].tolist() == want
    _ok()


@BOTH
@pytest.mark.parametrize("T,E,W,F,limit", [(1, 8, 128, 64, 1.0), (5, 16, 192, 128, 0.2), (130, 4, 64, 320, 7.0), (700, 3, 256, 192, 0.7), (1000, 12, 128, 512, 1.0)])
def test_gated_expert_products(dtype, T, E, W, F, limit):
    """Few rows per expert, experts without rows, and experts with several tiles of rows; every tile width and source of rows."""
    from relax_b200 import ops
    from relax_b200.ops import cuda as C

    h = _rand(1, T, W, dtype=dtype)
    gate, up, down = _rand(2, E, F, W, dtype=dtype) / W ** 0.5, _rand(5, E, F, W, dtype=dtype) / W ** 0.5, _rand(3, E, W, F, dtype=dtype) / F ** 0.5
    z = _rand(4, T, 64)
    z[:, 0] += 2.0                     # one expert takes most rows
    plan = ops.moe_route(z, _moe(E, 2, 2, F, limit=limit), dtype, None, torch.zeros(E + 2, dtype=dtype, device="cuda"))
    ex = plan.expert.cpu()
    flat = (plan.offset.cpu()[ex.clamp(max=E - 1).long()] + plan.place.cpu()).long()
    want = torch.zeros(int((ex < E).sum()), W, dtype=F64)
    d = lambda x: x.to(F64).cpu()
    for e in range(E):
        t, j = (ex == e).nonzero(as_tuple=True)
        want[flat[t, j]] = O.expert(d(h)[t], d(gate[e]), d(up[e]), d(down[e]), limit)
    rows = ops.glu_rows(gate, up)
    plans = [(bn, full) for bn in (128, 256) for full in (False, True)] if dtype == BF else [(128, False)]
    keep = C._moe_plan
    try:
        for choice in plans:
            C._moe_plan = lambda *a, choice=choice: choice
            got = ops.moe_experts(h, plan, rows, down, "clamped_swish", limit)
            if len(want):
                _close(got[: len(want)], want, 2e-2 if dtype == BF else 1e-5)
    finally:
        C._moe_plan = keep
    _ok()


@BOTH
@pytest.mark.parametrize("width,top,I", [(4096, 8, 4), (90, 2, 3), (74, 1, 20), (2048, 6, 0)])
def test_norm_of_the_sum(dtype, width, top, I):
    from relax_b200 import ops

    T, E, pitch, alpha, eps = 33, 16, (width + 63) // 64 * 64, 1.6, 1e-3
    plan = ops.moe_route(_rand(7, T, 64), _moe(E, I, top, 8), dtype, None, torch.zeros(E + I, dtype=dtype, device="cuda"))
    rows, y = _rand(1, T * top, pitch, dtype=dtype), _rand(2, T, pitch, dtype=dtype)
    w, b, fw, fb = (_rand(s, pitch, dtype=dtype) for s in (3, 4, 5, 6))
    for x in (rows, y, w, b, fw, fb):
        x[..., width:] = 0
    real = plan.expert < E
    rows[int(real.sum()):] = float("nan")              # rows behind the last one are nobody's
    flat = torch.where(real, plan.offset[plan.expert.clamp(max=E - 1).long()] + plan.place, 0).long()
    pw = plan.weight.to(F64)
    z = (rows[flat].to(F64) * (pw * real)[..., None]).nan_to_num(0.0).sum(1)[:, :width]
    d = lambda x: x[..., :width].to(F64)
    base = _rand(8, T, pitch) + 5.0
    base[:, width:] = 0
    for shared in (y, None):
        for experts in ((rows, plan), None):
            if shared is None and experts is None:
                continue
            for nxt in (None, (fw, fb)):
                total = alpha * d(base)
                if experts:
                    total = total + z + d(base) * (pw * ~real).sum(1, keepdim=True)
                if shared is not None:
                    total = total + d(shared)
                res = base.clone()
                h = ops.sum_norm(res, shared, w, b, width, alpha, eps, nxt, 0.3, experts)
                want = O.centred(total, d(w), d(b), eps)
                _close(res[:, :width], want, 1e-5)
                _close(h[:, :width], want if nxt is None else O.centred(want, d(fw), d(fb), eps) * 0.3, 5e-3 if dtype == BF else 1e-5)
                assert not h[:, width:].any() and not res[:, width:].any()
    res = base.clone()
    ops.sum_norm(res, y, w, None, width, alpha, eps)
    _close(res[:, :width], O.rms(alpha * d(base) + d(y), d(w), eps), 1e-5)
    # identity experts in the norm of the output alone: their output is the stream
    res = base.clone()
    ops.norm_add(res, None, w, width, 1, eps, None, (rows, plan))
    _close(res[:, :width], d(base) + O.rms(z + d(base) * (pw * ~real).sum(1, keepdim=True), d(w), eps), 1e-5)
    _ok()


@BOTH
def test_embedded_tokens_are_scaled(dtype):
    from relax_b200 import ops

    table = _rand(1, 50, 192, dtype=dtype)
    tok = torch.tensor([3, 49, 0, 3], device="cuda")
    res, h = ops.embed_rows(tok, table, scale=0.7)
    _close(res, table[tok].to(F64) * 0.7, 1e-7)
    assert torch.equal(h, res.to(dtype))
    _ok()


# ---------------------------------------------------------------------------------------------------- engine


def _agrees(got, case, dtype):
    """fp32: every row.  bf16: rows whose expert choices are not close calls, within what rounding does."""
    want, gaps, _ = case
    d = distances(got, want)
    if dtype == torch.float32:
        d = d[gaps > 1e-6]
        assert float(d.max()) < 1e-4, float(d.max())
    else:
        sure = d[gaps > 0.01]
        assert len(sure) >= min(4, len(d) // 2)
        # a row that did take another expert changes what later rows read of it
        assert float(sure.median()) < 0.03 and float(sure.quantile(0.9)) < 0.12, (float(sure.median()), float(sure.quantile(0.9)), float(sure.max()))


@BOTH
@pytest.mark.parametrize("name", list(O.CONFIGS))
def test_schedules_agree_with_the_plain_model(name, dtype):
    cfg, t = O.random_model(O.CONFIGS[name], 1)
    toks = tokens(cfg, 75, 1)
    case = O.run(cfg, t, toks)
    eng = D.engine(cfg, t, "cuda", dtype, blocks=6)
    for sizes in ([75], [1], [2], [17, 1, 3, 30], [64, 1, 1]):
        _agrees(D.feed_alone(eng, toks, sizes), case, dtype)
        D.all_free(eng)
    _ok()


def test_residual_stream_after_every_layer():
    cfg, t = O.random_model(O.CONFIGS["even"], 3)
    toks = tokens(cfg, 30, 1)
    want = O.run(cfg, t, toks)[2]
    for dtype, tol in ((torch.float32, 1e-5), (BF, 5e-2)):
        eng = D.engine(cfg, t, "cuda", dtype, blocks=6)
        r, taps = eng.open_sequence(), []
        r.prompt.extend(toks)
        eng.run_segments([(r, 30)], [[]], taps)
        assert len(taps) == len(want)
        if dtype == torch.float32:
            for a, b in zip(taps, want):
                _close(a, b, tol)
        else:
            assert float((taps[0].to(F64).cpu() - want[0]).pow(2).mean().sqrt()) < tol
    _ok()


@BOTH
def test_long_prompts_in_portions_beside_other_requests(dtype):
    """Contexts of several tiles and windows, requests that join and leave, few pages and slots."""
    cfg, t = O.random_model(O.CONFIGS["even"], 2)
    seqs = [tokens(cfg, n, n) for n in (310, 30, 200, 3, 133)]
    cases = [O.run(cfg, t, s) for s in seqs]
    eng = D.engine(cfg, t, "cuda", dtype, blocks=50)
    for sizes in ([310], [200, 1, 93, 2], [131, 3], [64, 192]):
        _agrees(D.feed_alone(eng, seqs[0], sizes), cases[0], dtype)
    got = D.feed_mixed(eng, seqs, [[193, 1, 100], [1], [0, 130, 5], [2, 1], [16, 0, 31, 2]], [0, 0, 1, 2, 33])
    for g, c in zip(got, cases):
        _agrees(g, c, dtype)
    D.all_free(eng)
    _ok()


def test_long_portions_of_every_head_width():
    """Portions that project the keys and values of their whole context: heads below, at and above 128 features."""
    for heads, dim, rot, vdim, rank in ((3, 10, 6, 7, 20), (4, 64, 64, 96, 64), (2, 128, 64, 128, 128), (2, 130, 32, 40, 64), (2, 200, 32, 24, 64)):
        cfg, t = O.random_model(O.stack(96, 131, 1e-5, [O.lat(heads, dim, rot, vdim, rank, 2.0 / (dim + rot) ** 0.5, 1e3),
                                                       O.lat(heads, dim, rot, vdim, rank, 2.0 / (dim + rot) ** 0.5, 1e3)]), 3)
        seqs = [tokens(cfg, n, n) for n in (420, 205)]
        want = [O.model(cfg, t, s) for s in seqs]
        eng = D.engine(cfg, t, "cuda", BF, blocks=60)
        for sizes in ([420], [5, 250, 1], [193, 227]):
            assert distance(D.feed_alone(eng, seqs[0], sizes), want[0]) < 0.05, (dim, sizes)
        for g, w in zip(D.feed_mixed(eng, seqs, [[192, 3, 225], [200, 1]], [0, 0]), want):
            assert distance(g, w) < 0.05, dim
    _ok()


def test_bf16_rows_do_not_depend_on_portions_batch_or_pages():
    cfg, t = O.random_model(O.CONFIGS["odd"], 8)
    toks = tokens(cfg, 150, 3)
    eng = D.engine(cfg, t, "cuda", BF, blocks=40)
    gaps = O.run(cfg, t, toks)[1]
    a = D.feed_alone(eng, toks, [150]).to(F64)
    other = [tokens(cfg, n, n) for n in (33, 90)]
    for b in (D.feed_alone(eng, toks, [2]), D.feed_alone(eng, toks, [97, 1, 1]), D.feed_mixed(eng, [toks] + other, [[31, 2, 1], [7], [20, 1]], [0, 1, 2])[0]):
        d = distances(b, a)[gaps > 0.01]
        assert float(d.median()) < 0.02 and float(d.quantile(0.9)) < 0.08, (float(d.median()), float(d.quantile(0.9)), float(d.max()))
    _ok()


def test_a_far_token_decides_in_prompts_and_in_decoding():
    """Scales so large that single keys take whole rows, from far back and across portions."""
    cfg, t = O.random_model(O.stack(64, 90, 1e-6, [O.lat(2, 16, 8, 24, 32, 0.5, 1e4), O.att(2, 1, 16, 40, 0.5, 4, 1e4, 300), O.lat(2, 16, 8, 24, 32, 0.5, 1e4)]), 3, sharp=8.0)
    toks = tokens(cfg, 900, 1)
    want, gaps, _ = O.run(cfg, t, toks)
    eng = D.engine(cfg, t, "cuda", torch.float32, blocks=60)
    for sizes in ([900], [860] + [1] * 40, [37, 3]):
        d = distances(D.feed_alone(eng, toks, sizes), want)
        assert float(d.quantile(0.99)) < 2e-3, (sizes, float(d.max()))
    _ok()


def test_long_decoding():
    cfg, t = O.random_model(O.CONFIGS["odd"], 4)
    toks = tokens(cfg, 300, 1)
    case = O.run(cfg, t, toks)
    eng = D.engine(cfg, t, "cuda", torch.float32, blocks=20)
    _agrees(D.feed_alone(eng, toks, [1]), case, torch.float32)
    _ok()


@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation_on_the_gpu(graph):
    from relax_b200.rollout.engine import SamplingParams

    cfg, t = O.random_model(O.CONFIGS["odd"], 5)
    prompts = [tokens(cfg, n, 40 + n) for n in (3, 70, 17, 9, 1)]
    want = [D.greedy(cfg, t, p, 12) for p in prompts]
    eng = D.engine(cfg, t, "cuda", torch.float32, blocks=40, state_slots=3, max_prefill_tokens=40, use_cuda_graph=graph, max_model_len=128, decode_window=5)
    res = eng.generate(prompts + [prompts[1]] * 2, SamplingParams(temperature=0.0, max_new_tokens=12, ignore_eos=True), group_keys=[0, 1, 2, 3, 4, 1, 1])
    assert [r.output for r in res] == want + [want[1]] * 2
    assert bool(eng.stats.get("graph_replays", 0)) == graph
    eng.close()
    _ok()


def test_bf16_captured_windows_equal_host_driven_steps():
    from relax_b200.models.config import get_config
    from relax_b200.rollout.engine import RolloutEngine, SamplingParams

    specs = get_config("zupupel-15b").layer_specs[:3]
    outs = []
    for graph in (False, True):
        eng = RolloutEngine(get_config("zupupel-15b", num_layers=3, layer_specs=specs, vocab_size=2000), device="cuda", num_kv_blocks=60, block_size=64,
                            use_cuda_graph=graph, max_model_len=512, state_slots=8)
        eng.weights.flat.normal_(0, 0.03, generator=torch.Generator(device="cuda").manual_seed(3))
        g = torch.Generator().manual_seed(0)
        prompts = [torch.randint(0, 2000, (n,), generator=g).tolist() for n in (5, 40, 230, 33, 64)]
        outs.append(eng.generate(prompts, SamplingParams(max_new_tokens=20, ignore_eos=True)))
        eng.close()
        _ok()
    same = sum(a.output == b.output for a, b in zip(*outs))
    assert same >= 4, same      # (a sampled token may sit on the edge of two)


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_program(tmp_path, dtype):
    from relax_b200.models import zupupel

    cfg, t = O.random_model(O.CONFIGS["wide"], 6)
    zupupel.save(str(tmp_path / "m"), zupupel.config_from_dict(cfg), t)
    a, b = tokens(cfg, 50, 1), tokens(cfg, 20, 2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [29, 3]}, {"id": "y", "tokens": b, "want": [19]}], "end": ["y"]},
             {"step": 1, "entries": [{"id": "x", "tokens": a[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[31:], "want": [18]}, {"id": "z", "tokens": b[:2], "want": [0, 1]}], "end": ["x", "z"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    wa, wb = O.run(cfg, t, a), O.run(cfg, t, b)
    for name, rows in (("0", [(wa, 29), (wa, 3), (wb, 19)]), ("2", [(wa, 49), (wb, 0), (wb, 1)])):
        got = torch.frombuffer(bytearray((tmp_path / f"{name}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        for z, (w, i) in zip(got, rows):
            if dtype == "float32" or w[1][i] > 0.01:
                assert distance(z[None], w[0][i:i + 1]) < (0.1 if dtype == "bfloat16" else 1e-4)
