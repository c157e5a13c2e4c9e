"""Zoguzen stacks: every mechanism, the reader, cache, scheduler and generation on the CPU against plain float64 statements."""
import io
import json
import os
import sys
from types import SimpleNamespace

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import composed_driver as D  # noqa: E402
import oracle_zoguzen as O  # noqa: E402
from oracle_composed import distance, tokens  # noqa: E402

F64 = torch.float64
TIGHT = 2e-5


def _close(got, want, tol):
    err = (got.to(F64) - want.to(F64)).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), (err, want.abs().max().item())


def _rand(seed, *s):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


def _batch(lens, starts, slots):
    """Segments of ``lens`` rows that begin at positions ``starts`` of their sequences."""
    cu = [0]
    for n in lens:
        cu.append(cu[-1] + n)
    return SimpleNamespace(cu=torch.tensor(cu), ctx=torch.tensor([a + n for a, n in zip(starts, lens)]), state_slot=torch.tensor(slots))


# ---------------------------------------------------------------------------------------------------- mechanisms alone


def test_convolved_projections_keep_their_last_rows():
    """Biases, taps, norms head by head and rotation; a sequence in portions equals the whole, also when its slot held another one's rows."""
    from relax_b200 import ops

    H, G, dim, vdim, rot, n, eps = 4, 2, 10, 7, 6, 4, 1e-2
    C, T = H * dim + G * (dim + vdim), 9
    x, bias, taps = _rand(1, T, C + 3), _rand(2, C), _rand(3, C, n)
    qw, kw = 1 + _rand(4, dim), 1 + _rand(5, dim)
    f = [0.7, 0.2, 0.01]
    u = O.convolved(x[:, :C].to(F64) + bias.to(F64), taps.to(F64))
    q, k, v = u.split([H * dim, G * dim, G * vdim], 1)
    want_q = O.turned(O.rms(q.view(T, H, dim), qw.to(F64), eps), range(T), f)
    want_k = O.turned(O.rms(k.view(T, G, dim), kw.to(F64), eps), range(T), f)
    for sizes in ([9], [2, 1, 1, 5], [1] * 9, [3, 6]):
        state, kp, vp, at, got = _rand(6, 3, n - 1, C), torch.zeros(T, G, 16), torch.zeros(T, G, 8), 0, []
        for m in sizes:
            b = _batch([m], [at], [2])
            b.slots = torch.arange(at, at + m)
            table = ops.rope_table(b.slots.int(), 0, torch.tensor(f, dtype=F64))
            got.append(ops.conv_inputs(x[at:at + m], bias, taps, state, b, qw, kw, table, H, G, dim, vdim, 16, rot, eps, kp, vp))
            at += m
        got = torch.cat(got)
        _close(got[..., :dim], want_q, 2e-6)
        _close(kp[..., :dim], want_k, 2e-6)
        _close(vp[..., :vdim], v.view(T, G, vdim), 2e-6)
        assert not got[..., dim:].any()
        assert torch.equal(state[2], x[T - n + 1:, :C]) and torch.equal(state[:2], _rand(6, 3, n - 1, C)[:2])


@pytest.mark.parametrize("base,dims,scaling", [(300.0, 12, (3.0, 1.0, 3.0, 60.0)), (1e4, 32, (8.0, 1.0, 4.0, 64.0)), (50.0, 8, None), (1e6, 64, (2.0, 0.5, 5.0, 100.0))])
def test_stretched_frequencies(base, dims, scaling):
    from relax_b200.models.config import LayerSpec
    from relax_b200.rollout.composed import ComposedForward

    rot = {"dims": dims, "base": base}
    if scaling:
        rot["scaling"] = dict(zip(("factor", "low", "high", "original"), scaling))
    want = torch.tensor(O.frequencies(rot), dtype=F64)
    spec = LayerSpec("attention", heads=1, dim=dims, vdim=4, kv_heads=1, rot_dims=dims, rot_base=base, rot_scaling=scaling)
    got = ComposedForward.rope_frequencies(SimpleNamespace(device="cpu"), spec)
    assert (got / want - 1).abs().max() < 1e-12
    if scaling:      # all three ranges occur
        plain = torch.tensor(O.frequencies({"dims": dims, "base": base}), dtype=F64)
        ratio = got / plain
        assert (ratio == 1).any() and (abs(ratio * scaling[0] - 1) < 1e-9).any() and ((ratio < 0.999) & (ratio * scaling[0] > 1.001)).any()


def _pools(lens, G, dim, vdim, page, seed):
    g = torch.Generator().manual_seed(seed)
    nb = [-(-L // page) for L in lens]
    perm = torch.randperm(sum(nb) + 2, generator=g).tolist()
    bt = torch.zeros(len(lens), max(nb) + 1, dtype=torch.int32)
    for s, n in enumerate(nb):
        bt[s, :n] = torch.tensor([perm.pop() for _ in range(n)])
    rows = [torch.tensor([int(bt[s, p // page]) * page + p % page for p in range(L)]) for s, L in enumerate(lens)]
    return torch.randn((sum(nb) + 2) * page, G, dim, generator=g), torch.randn((sum(nb) + 2) * page, G, vdim, generator=g), bt, rows


@pytest.mark.parametrize("kind,size,keep,cap,one,talk", [("window", 1, 0, 0.0, False, False), ("window", 4, 3, 0.0, False, False), ("window", 5, 100, 2.0, False, True),
                                                          ("window", 3, 5, 0.0, True, False), ("chunk", 1, 0, 3.0, True, True), ("chunk", 4, 0, 0.5, True, True),
                                                          ("chunk", 5, 0, 0.0, False, True), ("chunk", 100, 0, 7.0, True, False)])
def test_attention_sees_windows_first_tokens_and_chunks(kind, size, keep, cap, one, talk):
    from relax_b200.ops import reference as ref

    H, G, dim, vdim, page, scale = 6, 2, 10, 7, 4, 0.8
    lens, ctx = [1, 3, 6], [5, 9, 6]
    k, v, bt, rows = _pools(ctx, G, dim, vdim, page, 3)
    q, mix = _rand(1, 10, H, dim), torch.eye(H) + 0.5 * _rand(2, H, H)
    got = ref.paged_attention(q, k, v, bt, page, torch.tensor(ctx), torch.tensor([0, 1, 4, 10]), scale, torch.zeros(H) if one else None, 8,
                              size if kind == "window" else 0, None, keep, size if kind == "chunk" else 0, cap, mix if talk else None).view(10, H, 8)
    sees = O.sees_window(size, keep) if kind == "window" else O.sees_chunk(size)
    at = 0
    for s, (n, L) in enumerate(zip(lens, ctx)):
        p = O.weights(q[at:at + n].to(F64), k[rows[s]].to(F64), L - n, scale, sees, cap or None, one)
        if talk:
            p = O.talked(p, mix.to(F64))
        _close(got[at:at + n, :, :vdim], O.applied(p, v[rows[s]].to(F64)), 1e-5)
        at += n
    assert not got[..., vdim:].any()


def test_running_means_follow_their_gates():
    from relax_b200 import ops

    width, T = 13, 11
    x, zb, xb = _rand(1, T, 3 * 16), _rand(2, 16), _rand(3, 16)
    part = lambda k: x[:, 16 * k:16 * k + width].to(F64)
    S = O.mingru(O.sigmoid(part(0) + zb[:width].to(F64)), part(1) + xb[:width].to(F64))
    want = S * O.silu(part(2))
    for sizes in ([11], [2, 9], [1] * 11):
        state, at, got = torch.full((2, 1, 1, 16), 9.0), 0, []
        for n in sizes:
            got.append(ops.mingru(x[at:at + n], zb, xb, state, _batch([n], [at], [1]), width))
            at += n
        got = torch.cat(got)
        _close(got[:, :width], want, 1e-6)
        _close(state[1, 0, 0, :width], S[-1], 1e-6)
        assert not got[:, width:].any() and (state[0] == 9).all()
    # gates that shut or open completely
    x[:, :16], x[:, 16:32] = 200.0 * torch.tensor([-1.0, 1.0] * 8), -300.0
    out = ops.mingru(x, 0 * zb, 0 * xb, torch.zeros(1, 1, 1, 16), _batch([T], [0], [0]), width)
    assert torch.isfinite(out).all() and not out[:, 0].any()


def test_linear_attention_decays_row_by_row():
    from relax_b200 import ops

    H, d, dv, tau, T, eps = 3, 5, 6, 3.0, 10, 1e-3
    qd, vd = H * d, H * dv
    rows, z, b, w = _rand(1, T, 56 + vd), _rand(2, T, 16) * 4, _rand(3, qd), 1 + _rand(4, dv)
    heads = lambda x: x.to(F64).view(T, H, -1)
    q, k, v, g = heads(rows[:, :qd]) * d ** -0.5, heads(rows[:, qd:2 * qd]), heads(rows[:, 2 * qd:2 * qd + vd]), rows[:, 56:56 + vd].to(F64)
    alpha = heads(O.sigmoid(z[:, :qd].to(F64) + b.to(F64)) ** (1 / tau))
    o, S = O.linear_attention(q, k, v, alpha)
    want = O.rms(o, w.to(F64), eps).reshape(T, -1) * O.silu(g)
    for sizes in ([10], [2, 7, 1], [1] * 10):
        state, at, got = torch.full((2, H, d, 8), 5.0), 0, []
        for n in sizes:
            c = _batch([n], [at], [1])
            got.append(ops.gla(rows[at:at + n], z[at:at + n], b, w, state, c.state_slot, c.ctx, c.cu if n > 1 else None, H, d, dv, 56, eps, tau))
            at += n
        got = torch.cat(got)
        _close(got[:, :vd], want, 1e-5)
        _close(state[1, ..., :dv], S, 1e-5)
        assert not got[:, vd:].any() and (state[0] == 5).all()
    z[:] = -5000.0      # rows that are forgotten at once
    out = ops.gla(rows, z, b, w, torch.zeros(1, H, d, 8), torch.tensor([0]), torch.tensor([T]), torch.tensor([0, T]), H, d, dv, 56, eps, tau)
    assert torch.isfinite(out).all()


@pytest.mark.parametrize("E,top", [(7, 2), (5, 5), (4, 1), (1, 1)])
def test_gated_experts_are_weighted_over_the_chosen_ones(E, top):
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    W, ff, T, eps = 24, 10, 30, 1e-4
    spec = MoESpec(experts=E, top=top, ff=ff, act="swiglu", score="softmax", renormalize=True)
    h, router = _rand(1, T, W), _rand(2, E, W)
    gate, up, down = _rand(4, E, ff, W), _rand(5, E, ff, W), _rand(6, E, W, ff)
    w = {"router": router, **{f"e{e}.{n}": x[e] for e in range(E) for n, x in (("gate", gate), ("up", up), ("down", down))}}
    want, _ = O.routed(h.to(F64), {k: x.to(F64) for k, x in w.items()}, {"router": {"experts": E, "top": top}})
    pad = lambda x, n, dim: torch.cat([x, torch.zeros(*x.shape[:dim], n - x.shape[dim], *x.shape[dim + 1:])], dim)
    plan = ops.moe_route(ops.linear_fp32(h, router), spec, torch.float32)
    rows = ops.moe_experts(h, plan, ops.glu_rows(pad(gate, 64, 1), pad(up, 64, 1)), pad(down, 64, 2), "swiglu")
    res = _rand(7, T, W)
    total = res.to(F64) + want
    n1, n2 = _rand(8, W), _rand(9, W)
    a, b = ops.stream_step(res, W, eps, None, None, (rows, plan), (n1, n2))
    _close(res, total, 1e-5)
    _close(a, O.centred(total, n1.to(F64), eps), 2e-5)
    _close(b, O.centred(total, n2.to(F64), eps), 2e-5)


def test_stream_steps_and_shifted_tokens():
    from relax_b200 import ops

    T, W, P, eps = 6, 21, 64, 1e-2
    d = lambda x: x[..., :W].to(F64)
    cols = torch.arange(P) < W
    res, y0, y1 = (_rand(s, T, P) * cols for s in (1, 2, 3))
    w0, w1, n1, n2, mu = (_rand(s, P) * cols for s in (4, 5, 6, 7, 8))
    res += 30.0 * cols                     # a mean that matters
    a = res.clone()
    x, = ops.stream_step(a, W, eps, [y0, y1], (w0, w1))
    want = d(res) + 0.5 * (O.rms(d(y0), d(w0), eps) + O.rms(d(y1), d(w1), eps))
    _close(a[:, :W], want, 1e-6)
    assert torch.equal(x, a)
    a = res.clone()
    ops.stream_step(a, W, eps, [y0], (w0,))
    _close(a[:, :W], d(res) + O.rms(d(y0), d(w0), eps), 1e-6)
    want = d(res) + d(y0)
    norms = O.centred(want, d(n1), eps), O.centred(want, d(n2), eps)
    for lens in ([6], [2, 4], [1] * 6, [3, 1, 2]):      # one sequence in portions; its state follows
        state, got, at = _rand(9, 2, P), [], 0
        for n in lens:
            h = ops.stream_step(res[at:at + n].clone(), W, eps, [y0[at:at + n]], None, None, (n1, n2), (mu, state, _batch([n], [at], [1])))
            _close(h[1][:, :W], norms[1][at:at + n], 1e-5)
            got.append(h[0])
            at += n
        _close(torch.cat(got)[:, :W], O.shifted(norms[0], d(mu)), 1e-5)
        _close(state[1, :W], norms[0][-1], 1e-5)
        assert torch.equal(state[0], _rand(9, 2, P)[0])


def test_second_embedding_and_capped_logits():
    from relax_b200 import ops

    dim, first, ids = 5, 10, torch.tensor([3, 8, 3])
    z, table = _rand(1, 3, 64) * 3, _rand(2, 9, 24)
    g = ops.side_gate(z, table, ids, first, dim)
    assert g.shape == (3, 8) and not g[:, dim:].any()
    _close(g[:, :dim], O.gelu(z[:, :dim].to(F64)) * table[ids][:, first:first + dim].to(F64), 1e-6)
    x = torch.tensor([[-1000.0, -3.0, 0.0, 1e-3, 3.0, 90.0]])
    _close(ops.softcap(x.clone(), 6.0), 6.0 * torch.tanh(x.to(F64) / 6.0), 1e-6)


# ---------------------------------------------------------------------------------------------------- models and schedules


@pytest.mark.parametrize("name", list(O.CONFIGS))
def test_prompt_portions_and_decoding_equal_the_plain_statement(name):
    cfg, t = O.random_model(O.CONFIGS[name], 1, sharp=2.0)
    toks = tokens(cfg, 41, 1)
    want = O.model(cfg, t, toks)
    eng = D.engine(cfg, t, blocks=6)
    for sizes in ([41], [1], [2], [16], [17, 1, 3], [2, 15, 1, 1]):
        assert distance(D.feed_alone(eng, toks, sizes), want) < TIGHT, sizes
        D.all_free(eng)


def test_mistakes_would_show():
    """The random models are sharp enough that a mechanism left out or done differently moves the logits far beyond the
    tolerance of the other tests (the mistakes are made in the plain statement)."""
    cfg, t = O.random_model(O.CONFIGS["odd"], 1, sharp=2.0)
    toks = tokens(cfg, 45, 1)
    want = O.model(cfg, t, toks)

    def other(layer=None, part=None, **changes):
        c = json.loads(json.dumps(cfg))
        m = c if layer is None else c["layers"][layer]["mixer"]
        (m if part is None else m[part]).update(changes)
        return distance(O.model(c, t, toks), want)

    assert other(logit_softcap=9.0) > 1e-2 and other(norm={"eps": 3e-2}) > 1e-3
    left = cfg["layers"][3]["mixer"]["left"]
    scaling = left["rot"]["scaling"]
    turn = lambda **kw: {"rot": {**left["rot"], **kw}}
    for layer, part, change in ((0, None, {"mask": {"size": 20}}), (0, None, {"mask": {"size": 22}}), (2, None, {"mask": {"size": 8}}), (4, None, {"mask": {"size": 32}}),
                                (0, None, {"softcap": 6.0}), (2, None, {"softcap": 4.0}), (4, None, {"scale": 1.5}), (3, "left", {"scale": 0.8}),
                                (3, "left", {"mask": {"size": 11, "keep_first": 5}}), (3, "left", {"mask": {"size": 13, "keep_first": 5}}),
                                (3, "left", {"mask": {"size": 12, "keep_first": 4}}), (3, "left", {"mask": {"size": 12, "keep_first": 6}}),
                                (3, "left", turn(base=330.0)), (3, "left", turn(scaling=None)), (3, "left", turn(scaling={**scaling, "factor": 4.0})),
                                (3, "left", turn(scaling={**scaling, "low": 1.4})), (3, "left", turn(scaling={**scaling, "high": 4.0})),
                                (3, "left", turn(scaling={**scaling, "original": 50.0})), (3, "right", {"tau": 4.0})):
        assert other(layer, part, **change) > 5e-4, (layer, part, change)

    def changed(**tensors):
        return distance(O.model(cfg, {**t, **tensors}, toks), want)

    for name in ("l0.mix.q.norm", "l2.mix.q.norm", "l4.mix.k.norm", "l3.mix.right.norm", "l0.norm1", "l1.norm2", "final.norm", "l3.mix.left.out", "l3.mix.right.out",
                 "l2.side.norm"):
        assert changed(**{name: torch.ones_like(t[name])}) > 1e-3, name
    for name in ("l0.mix.q.b", "l0.mix.k.b", "l4.mix.v.b", "l1.mix.z.b", "l1.mix.x.b", "l3.mix.right.a2.b", "l3.shift", "l0.shift", "l5.shift", "l3.mix.left.g",
                 "l3.mix.right.g", "l1.mix.g", "l4.side.gate"):
        assert changed(**{name: torch.zeros_like(t[name])}) > 1e-3, name
    for name in ("l0.mix.q.conv", "l2.mix.q.conv", "l4.mix.k.conv", "l5.mix.left.v.conv"):      # the oldest tap
        w = t[name].clone()
        w[:, 0] = 0
        assert changed(**{name: w}) > 1e-3, name
    assert changed(**{"l0.mix.talk": torch.eye(6).bfloat16()}) > 1e-3 and changed(**{"l2.mix.talk": t["l2.mix.talk"].T.contiguous()}) > 1e-3
    flip = lambda n: O.model(cfg, t, toks[:n] + [(toks[n] + 1) % cfg["vocab"]] + toks[n + 1:])[-1:]
    assert all(distance(flip(n), want[-1:]) > 1e-4 for n in (0, 1, 20, 43))            # far tokens count


def _one_layer(layer, seed=3, dim=8):
    """One attention layer whose inputs carry no shift, no second embedding, and one tap: a row follows exactly the tokens it sees."""
    cfg, t = O.random_model(O.stack(32, 50, 1e-5, [layer], 4, 30.0), seed)
    for k in t:
        if k.endswith("shift") or k.endswith("side.proj"):
            t[k] = torch.zeros_like(t[k])
        if k.endswith("right.out"):      # leaves the left side alone
            t[k] = torch.zeros_like(t[k])
    return cfg, t


@pytest.mark.parametrize("layer,edges", [
    (O.pair(O.left(2, 1, 8, 8, 0.05, 7, 3, 1, 4, 100.0), O.right(1, 4, 4, 2.0, 2)), ((23, True), (22, False), (3, False), (2, True), (0, True))),
    (O.att(2, 1, 8, 8, 0.05, 10, 20.0, 1), ((20, True), (28, True), (19, False), (10, False), (0, False))),
    (O.att(2, 1, 8, 8, 0.05, 29, 20.0, 1), ((28, False), (0, False)))])
def test_windows_first_tokens_and_chunks_end_where_they_should(layer, edges):
    """The last of 30 rows follows a change of a token that it sees, and nothing of one that it does not."""
    cfg, t = _one_layer(layer)
    toks = tokens(cfg, 30, 2)
    eng = D.engine(cfg, t, blocks=4)
    cuts = (("prompt", [30]), ("decode", [1]), ("portions", [2, 5]))
    base = {n: D.feed_alone(eng, toks, s)[-1:] for n, s in cuts}
    for place, seen in edges:
        x = list(toks)
        x[place] = (x[place] + 7) % cfg["vocab"]
        for n, s in cuts:
            moved = distance(D.feed_alone(eng, x, s)[-1:], base[n].to(F64))
            assert (moved > 1e-4) == seen and (seen or moved < 1e-6), (n, place, moved)


def test_unequal_requests_in_one_batch_equal_each_alone_and_slots_and_pages_are_used_again():
    cfg, t = O.random_model(O.CONFIGS["odd"], 2, sharp=2.0)
    seqs = [tokens(cfg, n, 10 + n) for n in (33, 5, 48, 2, 17, 20, 31, 1)]
    want = [O.model(cfg, t, s) for s in seqs]
    eng = D.engine(cfg, t, blocks=9)          # fewer pages than all sequences together need
    plans = [[7, 1], [1], [16, 2, 0, 3], [2], [0, 5], [3], [9, 1, 1], [1]]
    got = D.feed_mixed(eng, seqs, plans, [0, 0, 0, 1, 8, 12, 16, 17])
    for g, w in zip(got, want):
        assert distance(g, w) < TIGHT
    D.all_free(eng)


def test_long_decoding():
    cfg, t = O.random_model(O.CONFIGS["single"], 3, sharp=2.0)
    toks = tokens(cfg, 150, 4)
    assert distance(D.feed_alone(D.engine(cfg, t, blocks=12), toks, [1]), O.model(cfg, t, toks)) < TIGHT


def test_caches_of_the_layers():
    cfg, t = O.random_model(O.CONFIGS["odd"], 2)
    eng = D.engine(cfg, t, blocks=4)
    kv = eng.kv
    assert kv.kv[2][0] is kv.kv[0][0] and (3, 0) in kv.kv and (3, 1) in kv.state and kv.state[1].shape == (5, 1, 1, 40) and len(kv.paged) == 8
    assert {k: tuple(x.shape[1:]) for k, x in kv.conv.items()} == {0: (2, 6 * 18 + 2 * 31), 2: (3, 6 * 18), (3, 0): (1, 40 + 2 * 17), 4: (4, 35 + 5 * 16), (5, 0): (2, 24 + 57)}
    assert len(kv.shift) == 6 and len(kv.slotted) == 3 + 5 + 6


@pytest.mark.parametrize("windowed", [False, True])
def test_greedy_generation_through_the_scheduler(windowed):
    from relax_b200.rollout.engine import SamplingParams

    cfg, t = O.random_model(O.CONFIGS["odd"], 4)
    prompts = [tokens(cfg, n, 40 + n) for n in (3, 30, 17, 9, 1)]
    want = [D.greedy(cfg, t, p, 6) for p in prompts]
    # two state slots: requests queue; 11 prompt tokens per step: prompts are cut beside decoding requests
    eng = D.engine(cfg, t, blocks=12, state_slots=2, max_prefill_tokens=11, windowed_decode=windowed, decode_window=3)
    res = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=6, ignore_eos=True))
    assert [r.output for r in res] == want
    assert all(len(r.logprobs) == 6 and max(r.logprobs) <= 1e-6 for r in res)
    assert eng.sm.num_free == eng.sm.n - 1 and eng.bm.num_free == eng.bm.num_blocks - (1 if windowed else 0)


def test_group_members_share_the_prompt_and_partial_rollouts_resume():
    from relax_b200.rollout.engine import SamplingParams

    cfg, t = O.random_model(O.CONFIGS["odd"], 5)
    p = tokens(cfg, 37, 3)
    want = D.greedy(cfg, t, p, 4)
    eng = D.engine(cfg, t, blocks=40, max_prefill_tokens=16)
    res = eng.generate([p] * 4, SamplingParams(temperature=0.0, max_new_tokens=4, ignore_eos=True), group_keys=[7] * 4)
    assert [r.output for r in res] == [want] * 4
    assert [r.cached_tokens for r in res] == [0, 32, 32, 32] and eng.stats["prefill_tokens"] == 37
    eng.add_request(p, SamplingParams(temperature=0.0, max_new_tokens=4, ignore_eos=True), resume_output=want[:2])
    done = []
    while eng.has_work:
        done += eng.step()
    assert done[0].output == want
    D.all_free(eng)


# ---------------------------------------------------------------------------------------------------- reader


def _shapes(t):
    return {k: tuple(v.shape) for k, v in t.items()}


def test_checkpoint_round_trip_and_registry(tmp_path):
    from relax_b200.checkpoint import hf as H
    from relax_b200.entrypoints.serve import engine_config
    from relax_b200.models import zoguzen
    from relax_b200.models.config import get_config

    cfg, t = O.random_model(O.CONFIGS["odd"], 6)
    mc = zoguzen.config_from_dict(cfg, shapes=_shapes(t))
    assert zoguzen.config_to_dict(mc) == cfg
    assert _shapes(t) == zoguzen.tensor_shapes(mc)
    assert mc.num_parameters() == sum(v.numel() for v in t.values())
    zoguzen.save(str(tmp_path), mc, t)
    read = engine_config("tiny", str(tmp_path))
    assert read.layer_specs == mc.layer_specs and read.pre_norm and read.token_shift and read.side_dim == 5 and read.logit_softcap == 7.0
    assert [s.decay_rank for s in read.specs_with("gla")] == [3, 20]
    H.validate_against_hf(read, str(tmp_path))
    for other in (get_config("tiny-zoguzen"), read.__class__(**{**read.__dict__, "logit_softcap": 8.0})):
        with pytest.raises(ValueError, match="does not match"):
            H.validate_against_hf(other, str(tmp_path))
    eng = D.engine(cfg, t, blocks=4)
    H.load_hf_into_rollout(str(tmp_path), read, eng.weights)
    toks = tokens(cfg, 9, 1)
    assert distance(D.feed_alone(eng, toks, [9]), O.model(cfg, t, toks)) < TIGHT


def test_loader_and_config_reject_what_does_not_fit():
    from relax_b200.models import zoguzen
    from relax_b200.models.config import LayerSpec, MoESpec, composed_config, get_config
    from relax_b200.models.transformer import GPTModel
    from relax_b200.rollout.engine import RolloutEngine

    cfg, t = O.random_model(O.CONFIGS["odd"], 7)
    for change in ({"l0.mix.extra": torch.zeros(2)}, {"embed": t["embed"][:-1]}, {"l2.mix.k": t["l0.mix.k"]}, {"l2.mix.k.conv": t["l0.mix.k.conv"]},
                   {"l3.mix.right.a2": t["l3.mix.right.a2"][:, :2]}):
        with pytest.raises(ValueError, match="does not fit"):
            D.engine(cfg, {**t, **change})
    with pytest.raises(ValueError, match="missing"):
        D.engine(cfg, {k: v for k, v in t.items() if k != "l1.shift"})

    def read(c):
        return zoguzen.config_from_dict(c, shapes=_shapes(t))

    def broken(layer, part=None, **mixer):
        c = json.loads(json.dumps(cfg))
        m = c["layers"][layer]["mixer"]
        (m if part is None else m[part]).update(mixer)
        return c

    with pytest.raises(ValueError, match="rank of the decay"):
        zoguzen.config_from_dict(cfg)
    with pytest.raises(ValueError, match="unknown mixer type"):
        read({**cfg, "layers": [{**cfg["layers"][0], "type": "lstm"}]})
    with pytest.raises(ValueError, match="feed-forward kind"):
        read({**cfg, "layers": [{**cfg["layers"][0], "mlp": {"kind": "dense", "ff": 8}}]})
    for bad in (broken(2, kv_from=2), broken(2, kv_from=1), broken(4, kv_from=3), broken(2, kv_heads=3)):
        with pytest.raises(ValueError, match="keys and values"):
            read(bad)
    for bad in (broken(0, conv=9), broken(0, softcap=-1.0)):
        with pytest.raises(ValueError, match="bad attention"):
            read(bad)
    with pytest.raises(ValueError, match="rotation scaling"):
        read(broken(3, "left", rot={"dims": 6, "base": 10.0, "scaling": {"factor": 2.0, "low": 4.0, "high": 4.0, "original": 9}}))
    with pytest.raises(ValueError, match="bad decay"):
        read(broken(3, "right", tau=0.0))
    one = dict(heads=1, dim=4, vdim=4, kv_heads=1)
    for kw in (dict(window=3, chunk=4), dict(keep_first=2), dict(sink=True, unit_sink=True), dict(talk=True, out_gate=True)):
        with pytest.raises(ValueError, match="attention layers see"):
            LayerSpec("attention", **one, **kw)
    with pytest.raises(ValueError, match="no other norm"):
        LayerSpec("attention", **one, conv=2, proj_norm=True)
    for kw in (dict(pair=None), dict(pair=(LayerSpec("mingru"),)), dict(pair=(LayerSpec("mingru", ff=8), LayerSpec("mingru")))):
        with pytest.raises(ValueError, match="pair"):
            LayerSpec("pair", **kw)
    with pytest.raises(ValueError, match="expert activation"):
        MoESpec(experts=2, top=1, ff=4, act="swiglu", limit=1.0)
    for layers, kw in (([LayerSpec("mingru", vdim=8)], dict(token_shift=True)), ([LayerSpec("mingru", vdim=8)], dict(side_dim=4)),
                       ([LayerSpec("mingru", vdim=8, ff=16)], dict(pre_norm=True)), ([LayerSpec("mingru", vdim=8)], dict(pre_norm=True, norm_sum=True))):
        with pytest.raises(ValueError):
            composed_config("x", layers, 8, 16, **kw)
    with pytest.raises(NotImplementedError, match="rollout engine"):
        GPTModel(get_config("tiny-zoguzen"))
    with pytest.raises(NotImplementedError):
        RolloutEngine(get_config("tiny-zoguzen"), return_routed_experts=True)
    assert get_config("zoguzen-15b").num_parameters() > 1.4e10


def test_mechanisms_mix_with_those_of_other_designs():
    """Layers of other kinds under norms in front, and without shift and second embedding: a batch equals each sequence alone."""
    from relax_b200.models.config import LayerSpec, MoESpec, composed_config
    from relax_b200.rollout.engine import RolloutEngine

    moe = MoESpec(experts=4, top=2, ff=24, act="relu2")
    layers = [LayerSpec("hgrn2", heads=2, dim=8, vdim=12), LayerSpec("latent_attention", heads=2, dim=8, vdim=8, kv_rank=16, scale=0.3, moe=moe),
              LayerSpec("pair", pair=(LayerSpec("mingru", vdim=20), LayerSpec("attention", heads=2, dim=8, vdim=8, kv_heads=1, scale=0.4, rot_dims=4, rot_base=100.0,
                                                                             qk_norm=True, sink=True, window=6)))]
    mc = composed_config("mixed", layers, hidden_size=32, vocab_size=40, pre_norm=True, tie_word_embeddings=True, dtype="fp32")
    eng = RolloutEngine(mc, device="cpu", dtype=torch.float32, num_kv_blocks=12, block_size=16, memory_saver=False, state_slots=4, use_cuda_graph=False)
    g = torch.Generator().manual_seed(1)
    for k, v in eng.weights.p.items():
        v.copy_(torch.randn(v.shape, generator=g) * (0.2 if v.dim() > 1 else 0.5))
    seqs = [[(7 * i + 3 * j) % 40 for j in range(n)] for i, n in enumerate((20, 9, 13))]
    alone = [D.feed_alone(eng, s, [len(s)]) for s in seqs]
    for g, w in zip(D.feed_mixed(eng, seqs, [[3, 1], [1], [5]], [0, 1, 0]), alone):
        assert distance(g, w.to(F64)) < TIGHT
    D.all_free(eng)


def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from relax_b200.entrypoints import trace
    from relax_b200.models import zoguzen

    cfg, t = O.random_model(O.CONFIGS["odd"], 9)
    zoguzen.save(str(tmp_path / "m"), zoguzen.config_from_dict(cfg, shapes=_shapes(t)), t)
    a, b = tokens(cfg, 20, 1), tokens(cfg, 6, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:9], "want": [8, 2]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": b, "want": [5]}, {"id": "a", "tokens": a[9:], "want": [10]}], "end": ["a", "c"]}]
    eng = trace.build_engine(str(tmp_path / "m"), torch.float32, 128, device="cpu")
    done = []
    trace.replay(eng, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), done.append)
    assert done == [0, 1, 2] and not (tmp_path / "1.f32").exists()
    wa, wb = O.model(cfg, t, a), O.model(cfg, t, b)
    for name, rows in (("0", [wa[8], wa[2]]), ("2", [wb[5], wa[19]])):
        got = torch.frombuffer(bytearray((tmp_path / f"{name}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert distance(got, torch.stack(rows)) < TIGHT
    D.all_free(eng)


def test_engine_server_serves_a_zoguzen_folder():
    from relax_b200.rollout.engine import SamplingParams
    from relax_b200.rollout.http_server import EngineServer, HTTPEngine

    cfg, t = O.random_model(O.CONFIGS["single"], 10)
    p = tokens(cfg, 11, 1)
    srv = EngineServer(D.engine(cfg, t, blocks=16))
    try:
        out = HTTPEngine(srv.url).generate([p], SamplingParams(temperature=0.0, max_new_tokens=4, ignore_eos=True))
        assert list(out[0].output) == D.greedy(cfg, t, p, 4)
    finally:
        srv.close() if hasattr(srv, "close") else srv.httpd.shutdown()
