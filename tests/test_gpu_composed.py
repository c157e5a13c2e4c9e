"""Composed stacks on a GPU: every kernel against a plain statement, the engine's schedules against each other and against
the float64 model, captured decode windows, and the trace program."""
import json
import os
import subprocess
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import composed_driver as D  # noqa: E402
import oracle_composed as O  # noqa: E402

pytestmark = pytest.mark.gpu
F64 = torch.float64
BOTH = pytest.mark.parametrize("dtype", [torch.bfloat16, torch.float32])


@pytest.fixture(autouse=True)
def _inference():
    with torch.no_grad():
        yield


def _gen(seed):
    return torch.Generator(device="cuda").manual_seed(seed)


def _rand(seed, *s, dtype=torch.float32):
    return torch.randn(*s, device="cuda", generator=_gen(seed)).to(dtype)


def _tol(dtype):
    return 2e-2 if dtype == torch.bfloat16 else 1e-5


def _close(got, want, tol):
    err = (got.to(F64) - want.to(F64)).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), (err, want.abs().max().item())


def _agrees(got, want, dtype):
    """fp32: every position.  bf16: the typical position, and no position beyond what rounding does to one whose read-out is
    nearly zero before its norm."""
    d = O.distances(got, want)
    if dtype == torch.float32:
        assert float(d.max()) < 1e-4, float(d.max())
    else:
        assert float(d.median()) < 0.02 and float(d.max()) < 0.15, (float(d.median()), float(d.max()))


def _ok():
    from relax_b200.ops import cuda as C

    torch.cuda.synchronize()
    C.check_error_flag()


# ---------------------------------------------------------------------------------------------------- kernels


@BOTH
@pytest.mark.parametrize("width,groups", [(4096, 8), (4096, 1), (90, 3), (360, 5), (200, 25), (64, 64)])
def test_norm_add(dtype, width, groups):
    from relax_b200 import ops

    pitch = (width + 63) // 64 * 64
    for next_w in (False, True):
        y, res = _rand(1, 7, pitch + 64, dtype=dtype)[:, :pitch], _rand(2, 7, pitch)
        w, nw = _rand(3, pitch, dtype=dtype), _rand(4, pitch, dtype=dtype)
        for x in (y, res, w, nw):
            x[..., width:] = 0
        want = res[:, :width].to(F64) + O.norm_in_groups(y[:, :width].to(F64), w[:width].to(F64), groups, 1e-3)
        h = ops.norm_add(res, y, w, width, groups, 1e-3, nw if next_w else None)
        _close(res[:, :width], want, 1e-6)
        _close(h[:, :width], O.norm_in_groups(want, nw[:width].to(F64), groups, 1e-3) if next_w else want, _tol(dtype) / 2 if dtype == torch.bfloat16 else 2e-6)
        assert h.dtype == dtype and not h[:, width:].any()


@BOTH
@pytest.mark.parametrize("act", ["silu", "gelu_tanh"])
def test_gated_unit(dtype, act):
    from relax_b200 import ops

    f = O.silu if act == "silu" else O.gelu_tanh
    gu = _rand(1, 33, 384, dtype=dtype) * 4
    gu[0, :4] = torch.tensor([-60.0, 60.0, 0.0, -9.0])
    g, u = gu.to(F64).chunk(2, -1)
    _close(ops.glu(gu, act), f(g) * u, _tol(dtype) / 2 if dtype == torch.bfloat16 else 1e-6)
    for T in (5, 100, 200):      # the fused decode GEMM, and the products behind it
        x, w = _rand(2, T, 192, dtype=dtype), _rand(3, 384, 192, dtype=dtype) / 8
        g, u = (x.to(F64) @ w.to(F64).T).chunk(2, -1)
        _close(ops.linear_glu(x, w, act), f(g) * u, _tol(dtype))
    _ok()


def _hgrn_case(dtype, H, dim, vdim, T, seed):
    x = _rand(seed, T, (2 * H * dim + H * vdim + 63) // 64 * 64, dtype=dtype)
    fb, lo, nw = _rand(seed + 1, H * dim, dtype=dtype), torch.rand(H * dim, device="cuda", generator=_gen(seed + 2)).to(dtype), _rand(seed + 3, vdim, dtype=dtype)
    lo[::4] = 0
    return x, fb, lo, nw


def _hgrn_plain(x, fb, lo, nw, H, dim, vdim, eps, S):
    x, fb, lo, nw = (t.to(F64).cpu() for t in (x, fb, lo, nw))
    out = []
    for t in range(x.shape[0]):
        q = O.silu(x[t, :H * dim]).view(H, dim)
        g = O.forget_gate(x[t, H * dim:2 * H * dim], fb, lo).view(H, dim)
        S, o = O.hgrn2_token(S, g, q, x[t, 2 * H * dim:2 * H * dim + H * vdim].view(H, vdim))
        out.append((O.rms(o, eps) * nw).reshape(-1))
    return torch.stack(out), S


@BOTH
@pytest.mark.parametrize("H,dim,vdim", [(2, 128, 128), (3, 40, 24), (1, 16, 40), (2, 33, 18), (5, 12, 7), (1, 200, 72), (2, 64, 130)])
def test_hgrn2_segments_and_steps(dtype, H, dim, vdim):
    """Segments of unequal length (one token to several chunks) in one launch, then single tokens, from states in shuffled
    slots; a segment at position 0 ignores what its slot holds."""
    from relax_b200 import ops

    eps, vp = 1e-5, (vdim + 3) // 4 * 4
    lens, before = [33, 1, 2, 16, 70, 17], [0, 5, 9, 0, 3, 0]
    T = sum(lens)
    x, fb, lo, nw = _hgrn_case(dtype, H, dim, vdim, T, 3)
    state = _rand(9, 8, H, dim, vp)
    state[..., vdim:] = 0
    slots = [6, 0, 3, 7, 1, 4]
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    S0 = [torch.zeros(H, dim, vdim, dtype=F64) if b == 0 else state[s, :, :, :vdim].to(F64).cpu() for s, b in zip(slots, before)]
    untouched = state[[2, 5]].clone()
    out = ops.hgrn2(x, fb, lo, nw, state, i32(slots), i32([b + n for b, n in zip(before, lens)]), i32(cu), H, dim, vdim, eps)
    assert torch.equal(untouched, state[[2, 5]])
    for s in range(len(lens)):
        want, S1 = _hgrn_plain(x[cu[s]:cu[s + 1]], fb, lo, nw, H, dim, vdim, eps, S0[s])
        _close(out[cu[s]:cu[s + 1], :H * vdim].cpu(), want, _tol(dtype) if dtype == torch.bfloat16 else 2e-5)
        _close(state[slots[s], :, :, :vdim].cpu(), S1, 2e-5)
        S0[s] = S1
    assert not out[:, H * vdim:].any() and not state[slots][..., vdim:].any()
    for _ in range(2):
        x1 = _rand(77, len(lens), x.shape[1], dtype=dtype)
        keep = [state[s, :, :, :vdim].to(F64).cpu() for s in slots]
        out = ops.hgrn2(x1, fb, lo, nw, state, i32(slots), i32([b + n + 1 for b, n in zip(before, lens)]), None, H, dim, vdim, eps)
        for s in range(len(lens)):
            want, S1 = _hgrn_plain(x1[s:s + 1], fb, lo, nw, H, dim, vdim, eps, keep[s])
            _close(out[s:s + 1, :H * vdim].cpu(), want, _tol(dtype) if dtype == torch.bfloat16 else 2e-5)
            _close(state[slots[s], :, :, :vdim].cpu(), S1, 1e-5)
    # a first token: zero state whatever the slot holds
    out = ops.hgrn2(x1, fb, lo, nw, state, i32(slots), i32([1] * len(lens)), None, H, dim, vdim, eps)
    want, S1 = _hgrn_plain(x1[2:3], fb, lo, nw, H, dim, vdim, eps, torch.zeros(H, dim, vdim, dtype=F64))
    _close(state[slots[2], :, :, :vdim].cpu(), S1, 1e-5)


@pytest.mark.parametrize("H,dim,vdim", [(2, 128, 128), (3, 48, 40), (1, 16, 128)])
def test_hgrn2_spans_side_by_side(H, dim, vdim):
    """Long segments cut into spans that run in parallel, beside segments of one span and of one token."""
    from relax_b200 import ops
    from relax_b200.rollout.composed import recurrent_spans

    eps, lens, before = 1e-5, [1, 230, 16, 97], [4, 11, 0, 0]
    x, fb, lo, nw = _hgrn_case(torch.bfloat16, H, dim, vdim, sum(lens), 31)
    lo = 1 - lo * 0.05                                 # gates near one: what a span inherits matters to its end
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    cuts = recurrent_spans(lens, H, ctas=10 ** 6, shortest=32)
    assert [b - a for a, b in zip(cuts[1], cuts[1][1:])] == [1, 5, 1, 3]
    state = _rand(9, 6, H, dim, (vdim + 3) // 4 * 4)
    slots = [3, 1, 5, 0]
    S0 = [torch.zeros(H, dim, vdim, dtype=F64) if b == 0 else state[s, :, :, :vdim].to(F64).cpu() for s, b in zip(slots, before)]
    out = ops.hgrn2(x, fb, lo, nw, state, i32(slots), i32([b + n for b, n in zip(before, lens)]), i32(cu), H, dim, vdim, eps, (i32(cuts[0]), i32(cuts[1])))
    for s in range(len(lens)):
        want, S1 = _hgrn_plain(x[cu[s]:cu[s + 1]], fb, lo, nw, H, dim, vdim, eps, S0[s])
        _close(out[cu[s]:cu[s + 1], :H * vdim].cpu(), want, 2e-2)
        _close(state[slots[s], :, :, :vdim].cpu(), S1, 2e-5)


@BOTH
def test_hgrn2_gates_at_their_ends(dtype):
    """Gates that close completely (the state is replaced at once) and that never close (the state is kept over hundreds of
    tokens), side by side; nothing overflows and old values neither leak nor vanish."""
    from relax_b200 import ops

    H, dim, vdim, T = 1, 64, 64, 600
    x, fb, lo, nw = _hgrn_case(dtype, H, dim, vdim, T, 21)
    fb.zero_()
    lo.zero_()
    x[:, dim:dim + 16] = -120.0              # gate 0
    x[:, dim + 16:dim + 32] = 120.0          # gate 1: nothing is written, nothing fades
    lo[48:] = 1.0                            # bound 1: likewise
    state = _rand(5, 2, H, dim, vdim)
    keep = state[1].clone()
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    out = ops.hgrn2(x, fb, lo, nw, state, i32([1]), i32([T + 4]), i32([0, T]), H, dim, vdim, 1e-5)
    want, S1 = _hgrn_plain(x, fb, lo, nw, H, dim, vdim, 1e-5, keep.to(F64).cpu())
    _close(out.cpu(), want, _tol(dtype) if dtype == torch.bfloat16 else 2e-5)
    _close(state[1].cpu(), S1, 2e-5)
    assert torch.equal(state[1, 0, 16:32], keep[0, 16:32]) and torch.equal(state[1, 0, 48:], keep[0, 48:])


@BOTH
def test_latent_write(dtype):
    from relax_b200 import ops

    for rank in (36, 64, 300):
        pitch = (rank + 63) // 64 * 64
        raw, w = _rand(1, 9, pitch + 128, dtype=dtype)[:, 64:64 + pitch], _rand(2, pitch, dtype=dtype)
        pool = torch.full((40, pitch), 7.0, dtype=dtype, device="cuda")
        slots = torch.tensor([3, 39, 0, 17, 16, 15, 31, 32, 8], device="cuda")
        ops.latent_write(raw, w, rank, 1e-4, pool, slots)
        _close(pool[slots, :rank], O.rms(raw[:, :rank].to(F64), 1e-4) * w[:rank].to(F64), _tol(dtype) / 2)
        assert not pool[slots, rank:].any()
        other = torch.ones(40, dtype=torch.bool)
        other[slots.cpu()] = False
        assert bool((pool[other.cuda()] == 7).all())


@BOTH
@pytest.mark.parametrize("T,H,K,N", [(1, 3, 24, 64), (5, 4, 128, 512), (130, 2, 40, 320), (300, 5, 64, 128)])
def test_head_linear(dtype, T, H, K, N):
    from relax_b200 import ops

    x = _rand(1, T, H * K + 64, dtype=dtype)[:, :H * K].view(T, H, K)
    w = _rand(2, H, K, N, dtype=dtype) / K ** 0.5
    _close(ops.head_linear(x, w, False), torch.einsum("thk,hkn->thn", x.to(F64), w.to(F64)), _tol(dtype))
    z = _rand(3, T, H, N, dtype=dtype)
    _close(ops.head_linear(z, w, True), torch.einsum("thn,hkn->thk", z.to(F64), w.to(F64)), _tol(dtype) * (N / K) ** 0.5)
    _ok()


def test_fp32_linear_is_true_fp32():
    from relax_b200 import ops

    for M, N, K in ((1, 64, 64), (70, 130, 33), (300, 512, 640)):
        x, w = _rand(1, M, K), _rand(2, N, K)
        want = x.to(F64) @ w.to(F64).T
        assert (ops.linear(x, w).to(F64) - want).abs().max() < 1e-5 * K ** 0.5


def _paged(lens_ctx, R, page, dtype, seed):
    """Latent rows of several sequences in shuffled pages, and the same rows in order."""
    nb = [(L + page - 1) // page for L in lens_ctx]
    perm = torch.randperm(sum(nb) + 3, generator=torch.Generator().manual_seed(seed)).tolist()
    pool = _rand(seed, (sum(nb) + 3) * page, R, dtype=dtype)
    bt = torch.zeros(len(nb), max(nb) + 2, dtype=torch.int32)
    for s, n in enumerate(nb):
        bt[s, :n] = torch.tensor([perm.pop() for _ in range(n)])
    rows = [torch.tensor([int(bt[s, p // page]) * page + p % page for p in range(L)], device="cuda") for s, L in enumerate(lens_ctx)]
    return pool, bt.cuda(), rows


def _batch(lens, ctx, bt, H):
    from relax_b200.rollout.composed import SegmentBatch, attention_items

    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device="cuda")
    if all(n == 1 for n in lens):
        return SegmentBatch(None, None, i32(ctx), bt, None, max_ctx=max(ctx))
    return SegmentBatch(None, None, i32(ctx), bt, None, cu=i32([0]), max_ctx=max(ctx), items={H: i32(attention_items(lens, ctx, H))},
                        row_seg=i32([s for s, n in enumerate(lens) for _ in range(n)]),
                        row_pos=i32([c - n + k for n, c in zip(lens, ctx) for k in range(n)]))


def _attend(q, pool, rows, lens, ctx, scale, gate):
    out, t = [], 0
    for s, (n, L) in enumerate(zip(lens, ctx)):
        c = pool[rows[s]].to(F64)
        for k in range(n):
            vis = c[: L - n + k + 1]
            p = torch.softmax(q[t].to(F64) @ vis.T * scale, -1)
            out.append(p @ vis * torch.sigmoid(gate[t].to(F64))[:, None])
            t += 1
    return torch.stack(out)


@BOTH
@pytest.mark.parametrize("H,R,page", [(4, 64, 16), (16, 128, 64), (32, 512, 16), (40, 320, 16), (70, 128, 32), (3, 448, 128), (8, 192, 16)])
@pytest.mark.parametrize("lens", [[1, 1, 1, 1, 1], [1, 7, 2, 60, 130]])
def test_latent_attention(dtype, H, R, page, lens):
    from relax_b200 import ops

    ctx = [1, 129, 700, 257, 300] if len(set(lens)) > 1 else [1, 128, 129, 1000, 16]
    pool, bt, rows = _paged(ctx, R, page, dtype, H + R)
    q, gate = _rand(5, sum(lens), H, R, dtype=dtype), _rand(6, sum(lens), H + 8, dtype=dtype)[:, :H]
    scale = 1.5 / R ** 0.5
    got = ops.latent_attention(q, pool, _batch(lens, ctx, bt, H), page, scale, gate)
    _close(got, _attend(q, pool, rows, lens, ctx, scale, gate), _tol(dtype))
    _ok()


@BOTH
@pytest.mark.parametrize("n", [1, 5])
def test_latent_attention_single_keys(dtype, n):
    """One key stands out for each row: the newest visible one, the one behind it (which must not be seen), the first of the
    sequence, keys on both sides of page and tile borders, and keys far away in a context of several splits."""
    from relax_b200 import ops

    H, R, page, L, scale = 2, 128, 16, 2000, 1.0
    for where in (0, 1, 15, 16, 127, 128, 129, 255, 256, 1023, 1024, L - n - 1, L - n, L - n + 1, L - 1):
        if where >= L:
            continue
        pool, bt, rows = _paged([L], R, page, dtype, 1)
        pool.mul_(0.1)
        q = _rand(2, n, H, R, dtype=dtype)
        pool[rows[0][where]] = (q[0, 0] * 0.3).to(dtype)
        q[:] = q[:1, :1]
        gate = torch.full((n, H), 30.0, dtype=dtype, device="cuda")
        got = ops.latent_attention(q, pool, _batch([n], [L], bt, H), page, scale, gate)
        want = _attend(q, pool, rows, [n], [L], scale, gate)
        _close(got, want, 1e-2 if dtype == torch.bfloat16 else 1e-5)
        for k in range(n):
            near = (got[k, 0].float() - pool[rows[0][where]].float()).abs().max() < 0.05
            assert bool(near) == (where <= L - n + k), (where, k)
    _ok()


def test_flash_with_unequal_widths_and_gate():
    from relax_b200 import ops
    from relax_b200.rollout.composed import query_blocks

    bf = torch.bfloat16
    for H, dk, dv in ((3, 24, 16), (2, 128, 128), (4, 56, 72), (2, 192, 128), (1, 136, 40)):
        lens, ctx = [200, 300], [450, 300]
        q, k, v = _rand(1, 500, H, dk, dtype=bf), _rand(2, 750, H, dk, dtype=bf), _rand(3, 750, H, dv, dtype=bf)
        g = _rand(4, 500, H, dtype=bf)
        cq, ck, tiles = (torch.tensor(x, dtype=torch.int32, device="cuda") for x in ([0, 200, 500], [0, 450, 750], query_blocks(lens, ctx, 128)))
        got = ops.dense_flash(q, k, v, ck[:2].contiguous(), tiles, 0.3, g).view(500, H, dv)
        wide = _rand(5, 500, H * dv + 24, dtype=bf)[:, 8:8 + H * dv]
        fine = ops.dense_flash(q, k, v, ck[:2].contiguous(), tiles, 0.3, wide, True).view(500, H, dv)
        bare = ops.dense_flash(q, k, v, ck[:2].contiguous(), tiles, 0.3).view(500, H, dv)
        _close(fine, bare.to(F64) * torch.sigmoid(wide.to(F64)).view(500, H, dv), 2e-2)
        o = 0
        for s in range(2):
            kk, vv, qq = k[ck[s]:ck[s + 1]].to(F64), v[ck[s]:ck[s + 1]].to(F64), q[cq[s]:cq[s + 1]].to(F64)
            sc = torch.einsum("ihd,jhd->hij", qq, kk) * 0.3
            i = torch.arange(lens[s], device="cuda")[:, None] + ctx[s] - lens[s]
            sc = sc.masked_fill(torch.arange(ctx[s], device="cuda")[None] > i, float("-inf"))
            want = torch.einsum("hij,jhd->ihd", torch.softmax(sc, -1), vv) * torch.sigmoid(g[o:o + lens[s]].to(F64))[..., None]
            _close(got[o:o + lens[s]], want, 2e-2)
            o += lens[s]
    _ok()


# ---------------------------------------------------------------------------------------------------- engine


@BOTH
@pytest.mark.parametrize("name", list(O.CONFIGS))
def test_schedules_agree_with_the_plain_model(name, dtype):
    cfg = O.CONFIGS[name]
    t = O.random_model(cfg, 1, sharp=2.0)
    toks = O.tokens(cfg, 75, 1)
    want = O.model(cfg, t, toks)
    eng = D.engine(cfg, t, "cuda", dtype, blocks=6)
    for sizes in ([75], [1], [2], [17, 1, 3, 30], [64, 1, 1]):
        _agrees(D.feed_alone(eng, toks, sizes), want, dtype)
        D.all_free(eng)
    _ok()


@BOTH
def test_long_prompts_in_portions_beside_other_requests(dtype):
    """Portions above and below the length from which keys and values are projected, contexts of several tiles, requests
    that join and leave, few pages and slots."""
    cfg = O.CONFIGS["even"]
    t = O.random_model(cfg, 2, sharp=2.0)
    seqs = [O.tokens(cfg, n, n) for n in (420, 30, 260, 3, 199)]
    want = [O.model(cfg, t, s) for s in seqs]
    eng = D.engine(cfg, t, "cuda", dtype, blocks=62)
    for sizes in ([420], [200, 1, 193, 2], [191, 3], [64, 192]):
        _agrees(D.feed_alone(eng, seqs[0], sizes), want[0], dtype)
    got = D.feed_mixed(eng, seqs, [[193, 1, 200], [1], [0, 192, 5], [2, 1], [16, 0, 31, 2]], [0, 0, 1, 2, 33])
    for g, w in zip(got, want):
        _agrees(g, w, dtype)
    D.all_free(eng)
    _ok()


def test_a_far_token_decides_in_prompts_and_in_decoding():
    """A single key that dominates the attention of the last tokens from far back: the logits change when it changes."""
    cfg = O.CONFIGS["single"]
    t = O.random_model(cfg, 3, sharp=30.0)
    toks = O.tokens(cfg, 900, 1)
    want = O.model(cfg, t, toks)
    eng = D.engine(cfg, t, "cuda", torch.float32, blocks=60)
    for sizes in ([900], [860] + [1] * 40, [37, 3]):
        assert O.distance(D.feed_alone(eng, toks, sizes), want) < 2e-3, sizes
    _ok()


def test_long_decoding_keeps_the_states():
    cfg = O.CONFIGS["odd"]
    t = O.random_model(cfg, 4)
    toks = O.tokens(cfg, 300, 1)
    want = O.model(cfg, t, toks)
    eng = D.engine(cfg, t, "cuda", torch.float32, blocks=20)
    assert O.distance(D.feed_alone(eng, toks, [1]), want) < 1e-4
    _ok()


@pytest.mark.parametrize("graph", [False, True])
def test_greedy_generation_on_the_gpu(graph):
    from relax_b200.rollout.engine import SamplingParams

    cfg = O.CONFIGS["odd"]
    t = O.random_model(cfg, 5)
    prompts = [O.tokens(cfg, n, 40 + n) for n in (3, 70, 17, 9, 1)]
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

    outs = []
    for graph in (False, True):
        eng = RolloutEngine(get_config("talizen-1b", num_layers=4, layer_specs=get_config("talizen-1b").layer_specs[:4], vocab_size=2000), device="cuda",
                            num_kv_blocks=200, use_cuda_graph=graph, max_model_len=512, state_slots=8)
        eng.weights.flat.normal_(0, 0.03, generator=_gen(3))
        g = torch.Generator().manual_seed(0)
        prompts = [torch.randint(0, 2000, (n,), generator=g).tolist() for n in (5, 40, 230, 33, 64)]
        outs.append(eng.generate(prompts, SamplingParams(max_new_tokens=20, ignore_eos=True)))
        eng.close()
        _ok()
    for a, b in zip(*outs):
        assert a.output == b.output and max(abs(x - y) for x, y in zip(a.logprobs, b.logprobs)) < 1e-4


@pytest.mark.parametrize("dtype", ["bfloat16", "float32"])
def test_trace_program(tmp_path, dtype):
    from relax_b200.models import talizen

    cfg = O.CONFIGS["wide"]
    t = O.random_model(cfg, 6)
    talizen.save(str(tmp_path / "m"), talizen.config_from_dict({"architecture": "Talizen", **cfg}), t)
    a, b = O.tokens(cfg, 50, 1), O.tokens(cfg, 20, 2)
    steps = [{"step": 0, "entries": [{"id": "x", "tokens": a[:30], "want": [29, 3]}, {"id": "y", "tokens": b, "want": [19]}], "end": ["y"]},
             {"step": 1, "entries": [{"id": "x", "tokens": a[30:31], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": a[31:], "want": [18]}, {"id": "z", "tokens": b[:2], "want": [0, 1]}], "end": ["x", "z"]}]
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    p = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path), "--max-tokens", "128"],
                       input="".join(json.dumps(s) + "\n" for s in steps), capture_output=True, text=True, timeout=300)
    assert p.returncode == 0, p.stderr[-2000:]
    assert [x for x in p.stdout.splitlines() if x.startswith("done")] == ["done 0", "done 1", "done 2"] and not (tmp_path / "1.f32").exists()
    wa, wb = O.model(cfg, t, a), O.model(cfg, t, b)
    for name, rows in (("0", [wa[29], wa[3], wb[19]]), ("2", [wa[49], wb[0], wb[1]])):
        got = torch.frombuffer(bytearray((tmp_path / f"{name}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert O.distance(got, torch.stack(rows)) < (0.06 if dtype == "bfloat16" else 1e-4)
