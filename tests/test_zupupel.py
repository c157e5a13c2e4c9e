"""Zupupel stacks: every mechanism, the reader, cache, scheduler and generation on the CPU against plain float64 statements."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import composed_driver as D  # noqa: E402
import oracle_zupupel as O  # noqa: E402
from oracle_composed import distance, tokens  # noqa: E402

F64 = torch.float64
TIGHT = 2e-5


def _close(got, want, tol):
    err = (got.to(F64) - want.to(F64)).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), (err, want.abs().max().item())


def _rand(seed, *s):
    return torch.randn(*s, generator=torch.Generator().manual_seed(seed))


# ---------------------------------------------------------------------------------------------------- mechanisms alone


@pytest.mark.parametrize("dim,vdim,rot,halves", [(18, 13, 10, True), (16, 16, 16, True), (12, 20, 4, False), (7, 5, 0, True)])
def test_projections_are_normed_whole_turned_and_written(dim, vdim, rot, halves):
    from relax_b200 import ops

    H, G, T, eps = 6, 2, 5, 1e-2
    x, qw, kw = _rand(1, T, H * dim + G * (dim + vdim) + 3), 1 + _rand(2, H * dim), 1 + _rand(3, G * dim)
    x[:, : dim] *= 5                     # heads of unequal size: a norm head by head would differ
    pos = torch.tensor([0, 1, 77, 1500, 30000], dtype=torch.int32)
    table = ops.rope_table(pos + 2, -2, torch.tensor([50.0 ** (-2 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F64)) if rot else None
    kp, vp = torch.zeros(40, G, 32), torch.zeros(40, G, 32)
    slots = torch.tensor([3, 39, 0, 17, 16])
    run = lambda q_w, k_w, e, *pools: ops.projection_inputs(x, q_w, k_w, table, H, G, dim, vdim, 32, rot, halves, e, *pools, slots)
    turn = O.turn_halves if halves else O.turn_neighbours
    q = run(qw, kw, eps, kp, vp)
    for got, a, n, w in ((q, 0, H, qw), (kp[slots], H * dim, G, kw)):
        want = O.rms(x[:, a:a + n * dim].to(F64), w.to(F64), eps).view(T, n, dim)
        _close(got[..., :dim], turn(want, pos.tolist(), rot, 50.0), 2e-6)
        assert not got[..., dim:].any()
    _close(vp[slots, :, :vdim], x[:, (H + G) * dim:(H + G) * dim + G * vdim].view(T, G, vdim), 0)
    assert torch.equal(run(qw, None, eps, None, None), q)
    _close(run(None, None, 0.0, None, None)[..., :dim], turn(x[:, : H * dim].to(F64).view(T, H, dim), pos.tolist(), rot, 50.0), 2e-6)


def _pools(lens, G, dim, vdim, page, seed):
    g = torch.Generator().manual_seed(seed)
    nb = [-(-L // page) for L in lens]
    perm = torch.randperm(sum(nb) + 2, generator=g).tolist()
    bt = torch.zeros(len(lens), max(nb) + 1, dtype=torch.int32)
    for s, n in enumerate(nb):
        bt[s, :n] = torch.tensor([perm.pop() for _ in range(n)])
    rows = [torch.tensor([int(bt[s, p // page]) * page + p % page for p in range(L)]) for s, L in enumerate(lens)]
    return torch.randn((sum(nb) + 2) * page, G, dim, generator=g), torch.randn((sum(nb) + 2) * page, G, vdim, generator=g), bt, rows


@pytest.mark.parametrize("window", [0, 1, 2, 4, 5, 8, 100])
def test_windowed_attention_with_a_gate(window):
    from relax_b200.ops import reference as ref

    H, G, dim, vdim, page, scale = 6, 2, 10, 7, 4, 0.8
    lens, ctx = [1, 3, 6], [5, 9, 6]
    k, v, bt, rows = _pools(ctx, G, dim, vdim, page, 3)
    q, gate = _rand(1, 10, H, dim), _rand(2, 10, H * 8 + 5)
    got = ref.paged_attention(q, k, v, bt, page, torch.tensor(ctx), torch.tensor([0, 1, 4, 10]), scale, None, 8, window, gate).view(10, H, 8)
    opened = O.sigmoid(gate[:, : H * 8].to(F64)).view(10, H, 8)[..., :vdim]
    at = 0
    for s, (n, L) in enumerate(zip(lens, ctx)):
        want = O.attend(q[at:at + n].to(F64), k[rows[s]].to(F64), v[rows[s]].to(F64), L - n, scale, window or None)
        _close(got[at:at + n, :, :vdim], want * opened[at:at + n], 1e-5)
        at += n
    assert not got[..., vdim:].any()


def test_latent_rows_carry_a_rotated_part():
    """Absorbed queries over cached rows equal per-head keys and values made from them."""
    from relax_b200 import ops
    from relax_b200.ops import reference as ref

    T, H, d, r, R, dv, eps = 9, 3, 5, 6, 11, 4, 1e-3
    x, w = _rand(1, T, H * (d + r) + R + r), 1 + _rand(2, R)
    uk, uv = _rand(3, H * d, R), _rand(4, H * dv, R)
    pos = torch.arange(T, dtype=torch.int32) + 40
    table = ops.rope_table(pos, 0, torch.tensor([20.0 ** (-2 * i / r) for i in range(r // 2)], dtype=F64))
    q, c, k_rot = (t.clone() for t in x.split([H * (d + r), R, r], 1))
    q = q.view(T, H, d + r)
    pool, slots = torch.full((32, 16 + 16), 7.0), torch.randperm(32)[:T]
    ops.latent_write(c, w, R, eps, pool, slots, (q, k_rot, table, 16, r, d))
    x = x.to(F64)
    want_q = x[:, : H * (d + r)].view(T, H, d + r)
    want_q = torch.cat([want_q[..., :d], O.turn_neighbours(want_q[..., d:], pos.tolist(), r, 20.0)], -1)
    want_c = O.rms(x[:, H * (d + r): H * (d + r) + R], w.to(F64), eps)
    want_k = O.turn_neighbours(x[:, None, H * (d + r) + R:], pos.tolist(), r, 20.0)[:, 0]
    _close(q, want_q, 1e-6)
    _close(pool[slots, :R], want_c, 1e-6)
    _close(pool[slots, 16:16 + r], want_k, 1e-6)
    assert not pool[slots, R:16].any() and not pool[slots, 16 + r:].any()
    keys, values = O.latent_keys_values(want_c, want_k, uk.to(F64), uv.to(F64), H)
    want = O.attend(want_q, keys, values, 0, 0.3)
    full = torch.zeros(H, d + r, 32)
    full[:, :d, :R], full[:, d + torch.arange(r), 16 + torch.arange(r)] = uk.view(H, d, R), 1.0
    rows = pool[slots]
    o = ref.latent_attention(ops.head_linear(q, full, False), rows, torch.zeros(1, 1, dtype=torch.int32), 16, torch.tensor([T]), torch.tensor([0, T]), 0.3, None, 16)
    uvp = torch.zeros(H, dv, 16)
    uvp[..., :R] = uv.view(H, dv, R)
    gate = _rand(6, T, H * dv)
    _close(ops.head_linear(o, uvp, True, gate), want * O.sigmoid(gate.to(F64)).view(T, H, dv), 1e-5)


@pytest.mark.parametrize("E,I,top,groups,keep", [(13, 2, 4, 5, 3), (8, 0, 8, 4, 4), (4, 2, 1, 6, 1), (7, 3, 4, 2, 1), (3, 6, 2, 1, 1), (2, 1, 3, 1, 1)])
def test_router_chooses_by_corrected_scores_and_weighs_by_scores(E, I, top, groups, keep):
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    spec = MoESpec(experts=E, top=top, ff=8, groups=groups, keep=keep, act="clamped_swish", limit=1.0, renormalize=True, score="softmax", correction=True,
                   identity=I, group_best=1)
    N = E + I
    z, corr = _rand(E, 80, N + 4) * 2, _rand(9, N) * 0.3 - 0.9      # choice scores are mostly negative
    z[0, :N], z[1, :N] = -300.0 * torch.arange(N), 12.0 - torch.arange(N)
    plan = ops.moe_route(z, spec, torch.float32, None, corr)
    for t in range(80):
        s = O.weigh(z[t, :N].to(F64))
        chosen, gap = O.choose((s + corr.to(F64)).tolist(), top, groups, keep)
        if gap > 1e-6:
            assert plan.index[t].tolist() == chosen
            total = sum(s[e] for e in chosen) + 1e-20
            assert all(abs(a - s[e] / total) < 1e-5 for a, e in zip(plan.weight[t].tolist(), chosen))


def test_the_best_expert_of_a_group_counts_and_chosen_scores_may_vanish():
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    base = dict(ff=8, act="clamped_swish", limit=1.0, renormalize=True, score="softmax", correction=True)
    z = torch.tensor([[4.0, -9.0, 3.9, 3.8]])
    pick = lambda best, corr: ops.moe_route(z, MoESpec(experts=4, top=1, groups=2, keep=1, group_best=best, **base), torch.float32, None,
                                            torch.tensor(corr)).index.tolist()
    assert pick(1, [0.0] * 4) == [[0]] and pick(2, [0.0] * 4) == [[2]]
    assert pick(1, [-5.0, -5.0, -6.0, -4.0]) == [[3]]                # all choice scores negative: groups that are out are not zero
    z = torch.tensor([[0.0, -500.0, -500.0, 0.0]])
    plan = ops.moe_route(z, MoESpec(experts=4, top=2, **base), torch.float32, None, torch.tensor([-2.0, 1.0, 1.0, -2.0]))
    assert sorted(plan.index[0].tolist()) == [1, 2] and plan.weight.tolist() == [[0.0, 0.0]]


@pytest.mark.parametrize("limit", [0.3, 1.0, 50.0])
def test_clamped_experts_and_identity_experts_meet_the_stream(limit):
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    W, E, ff, T, alpha, eps = 24, 6, 10, 40, 1.3, 1e-4
    spec = MoESpec(experts=E, top=3, ff=ff, groups=3, keep=2, act="clamped_swish", limit=limit, renormalize=True, score="softmax", correction=True,
                   identity=3, group_best=1)
    h, router, corr = _rand(1, T, W), _rand(2, E + 3, W), _rand(3, E + 3) * 0.2
    gate, up, down = _rand(4, E, ff, W), _rand(5, E, ff, W), _rand(6, E, W, ff)
    w = {"router": router, "correction": corr, **{f"e{e}.{n}": x[e] for e in range(E) for n, x in (("gate", gate), ("up", up), ("down", down))}}
    want, _ = O.routed(h.to(F64), {k: x.to(F64) for k, x in w.items()},
                       {"expert": {"limit": limit}, "router": {"experts": E, "top": 3, "groups": {"count": 3, "keep": 2}}})
    pad = lambda x, n, dim: torch.cat([x, torch.zeros(*x.shape[:dim], n - x.shape[dim], *x.shape[dim + 1:])], dim)
    plan = ops.moe_route(ops.linear_fp32(h, router), spec, torch.float32, None, corr)
    assert (plan.index >= E).any()
    rows = ops.moe_experts(h, plan, ops.glu_rows(pad(gate, 64, 1), pad(up, 64, 1)), pad(down, 64, 2), "clamped_swish", limit)
    nw, nb, fw, fb = (_rand(s, W) for s in (7, 8, 9, 10))
    d = lambda x: x.to(F64)
    for nxt in (None, (fw, fb)):
        res = h.clone()
        out = ops.sum_norm(res, None, nw, nb, W, alpha, eps, nxt, 0.7, (rows, plan))
        total = O.centred(alpha * d(h) + want, d(nw), d(nb), eps)
        _close(res, total, 2e-5)
        _close(out, total if nxt is None else O.centred(total, d(fw), d(fb), eps) * 0.7, 2e-5)


def test_norm_after_the_sum():
    from relax_b200 import ops

    T, W, P = 4, 21, 64
    d = lambda x: x[..., :W].to(F64)
    res, y, w, b = _rand(1, T, P), _rand(2, T, P), _rand(3, P), _rand(4, P)
    res[:, W:], y[:, W:], w[W:], b[W:] = 0, 0, 0, 0
    res += 30.0 * (torch.arange(P) < W)                     # a mean that matters
    want = O.centred(0.4 * d(res) + d(y), d(w), d(b), 1e-2)
    rms = O.rms(0.4 * d(res) + d(y), d(w), 1e-2)
    a, c = res.clone(), res.clone()
    h = ops.sum_norm(a, y, w, b, W, 0.4, 1e-2)
    _close(a[:, :W], want, 1e-4)
    _close(h[:, :W], want, 1e-4)
    ops.sum_norm(c, y, w, None, W, 0.4, 1e-2)
    _close(c[:, :W], rms, 1e-5)
    assert not h[:, W:].any()


def test_embedded_tokens_are_scaled():
    from relax_b200 import ops

    table = _rand(6, 9, 16).bfloat16()
    res, h = ops.embed_rows(torch.tensor([3, 8]), table, scale=0.3)
    _close(res, table[[3, 8]].to(F64) * 0.3, 1e-7)
    assert h.dtype == torch.bfloat16 and torch.equal(h, res.bfloat16())


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

    def other(layer=None, **changes):
        c = json.loads(json.dumps(cfg))
        (c if layer is None else c["layers"][layer]["mixer"]).update(changes)
        return distance(O.model(c, t, toks), want)

    assert other(postln_alpha=1.6) > 1e-2 and other(embedding={"scale": 0.7}) > 1e-3 and other(logit_scale=0.5) > 1e-2
    assert other(norm={"eps": 3e-2}) > 1e-3
    for layer, change in ((0, {"mask": {"size": 20}}), (0, {"mask": {"size": 22}}), (2, {"mask": {"size": 8}}), (2, {"mask": {"size": 10}}), (3, {"mask": {"size": 32}}),
                          (4, {"mask": {"size": 41}}), (0, {"rot": {"dims": 8, "base": 1e3}}), (0, {"rot": {"dims": 10, "base": 1.1e3}}), (0, {"scale": 0.6}),
                          (1, {"rot": {"dims": 6, "base": 280.0}}), (1, {"scale": 0.75})):
        assert other(layer, **change) > 1e-3, (layer, change)

    def changed(**tensors):
        return distance(O.model(cfg, {**t, **tensors}, toks), want)

    for name in ("l0.mix.q.norm", "l0.mix.k.norm", "l2.mix.q.norm", "l1.mix.dkv.norm", "l1.norm1", "l0.norm2", "final.norm"):
        assert changed(**{name: torch.ones_like(t[name])}) > 1e-3, name
    for name in ("l0.norm1.b", "l3.norm1.b", "l2.norm2.b", "final.norm.b", "l0.mlp.correction", "l1.mix.g", "l3.mix.g"):
        assert changed(**{name: torch.zeros_like(t[name])}) > 1e-3, name
    flip = lambda n: O.model(cfg, t, toks[:n] + [(toks[n] + 1) % cfg["vocab"]] + toks[n + 1:])[-1:]
    assert all(distance(flip(n), want[-1:]) > 1e-4 for n in (0, 1, 15, 16, 43))            # every token counts


def test_a_window_ends_where_it_should():
    """One layer; the last row follows a change of the oldest token in its window and nothing of the one before."""
    window = 7
    cfg, t = O.random_model(O.stack(32, 50, 1e-5, [O.att(2, 1, 8, 8, 0.5, 4, 100.0, window)]), 3, sharp=0.1)
    toks = tokens(cfg, 30, 2)
    eng = D.engine(cfg, t, blocks=4)
    base = {n: D.feed_alone(eng, toks, s)[-1:] for n, s in (("prompt", [30]), ("decode", [1]), ("portions", [2, 5]))}
    for place, seen in ((29 - window + 1, True), (29 - window, False), (29 - window - 1, False), (0, False)):
        x = list(toks)
        x[place] = (x[place] + 7) % cfg["vocab"]
        for n, s in (("prompt", [30]), ("decode", [1]), ("portions", [2, 5])):
            moved = distance(D.feed_alone(eng, x, s)[-1:], base[n].to(F64))
            assert (moved > 1e-3) == seen and (seen or moved < 1e-6), (n, place, moved)


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


def test_caches_of_the_layers():
    cfg, t = O.random_model(O.CONFIGS["odd"], 2)
    eng = D.engine(cfg, t, blocks=4)
    kv = eng.kv.kv
    assert kv[2][0] is kv[0][0] and kv[4][1] is kv[0][1] and kv[3][0] is not kv[0][0] and len(eng.kv.paged) == 5
    assert eng.kv.latent[1].shape == (64, 128)               # 20 features and 6 turned ones, each in a chunk of 64


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

    cfg, t = O.random_model(O.CONFIGS["single"], 5)
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


def test_checkpoint_round_trip_and_registry(tmp_path):
    from relax_b200.checkpoint import hf as H
    from relax_b200.entrypoints.serve import engine_config
    from relax_b200.models import zupupel
    from relax_b200.models.config import get_config

    cfg, t = O.random_model(O.CONFIGS["odd"], 6)
    mc = zupupel.config_from_dict(cfg)
    assert zupupel.config_to_dict(mc) == cfg
    assert {k: tuple(v.shape) for k, v in t.items()} == zupupel.tensor_shapes(mc)
    assert mc.num_parameters() == sum(v.numel() for v in t.values())
    zupupel.save(str(tmp_path), mc, t)
    read = engine_config("tiny", str(tmp_path))
    assert read.layer_specs == mc.layer_specs and read.norm_sum and read.sum_alpha == 1.7 and read.embed_scale == 0.8 and read.logit_scale == 0.6
    H.validate_against_hf(read, str(tmp_path))
    for other in (get_config("tiny-zupupel"), H.config_from_hf(str(tmp_path)).__class__(**{**read.__dict__, "logit_scale": 0.7})):
        with pytest.raises(ValueError, match="does not match"):
            H.validate_against_hf(other, str(tmp_path))
    eng = D.engine(cfg, t, blocks=4)
    H.load_hf_into_rollout(str(tmp_path), read, eng.weights)
    toks = tokens(cfg, 9, 1)
    assert distance(D.feed_alone(eng, toks, [9]), O.model(cfg, t, toks)) < TIGHT


def test_missing_groups_masks_and_rotations_mean_none():
    cfg, t = O.random_model(O.CONFIGS["single"], 6)
    c = json.loads(json.dumps(cfg))
    c["layers"][0]["mlp"]["router"].pop("groups")
    c["layers"][0]["mixer"].pop("mask")
    for i in (0, 2):
        c["layers"][i]["mixer"]["rot"] = None
    toks = tokens(cfg, 12, 1)
    assert distance(D.feed_alone(D.engine(c, t, blocks=4), toks, [5, 1]), O.model(c, t, toks)) < TIGHT


def test_loader_and_config_reject_what_does_not_fit():
    from relax_b200.models import zupupel
    from relax_b200.models.config import LayerSpec, MoESpec, composed_config, get_config
    from relax_b200.models.transformer import GPTModel
    from relax_b200.rollout.engine import RolloutEngine

    cfg, t = O.random_model(O.CONFIGS["odd"], 7)
    for change in ({"l0.mix.extra": torch.zeros(2)}, {"head": t["head"][:-1]}, {"l2.mix.k": t["l0.mix.k"]}, {"l2.mix.k.norm": t["l0.mix.k.norm"]}):
        with pytest.raises(ValueError, match="does not fit"):
            D.engine(cfg, {**t, **change})
    with pytest.raises(ValueError, match="missing"):
        D.engine(cfg, {k: v for k, v in t.items() if k != "l1.norm2.b"})

    def broken(layer, **mixer):
        c = json.loads(json.dumps(cfg))
        c["layers"][layer]["mixer"].update(mixer)
        return c

    with pytest.raises(ValueError, match="unknown mixer type"):
        zupupel.config_from_dict({**cfg, "layers": [{**cfg["layers"][0], "type": "conv"}]})
    with pytest.raises(ValueError, match="feed-forward kind"):
        zupupel.config_from_dict({**cfg, "layers": [{**cfg["layers"][0], "mlp": {"kind": "dense", "ff": 8}}]})
    for bad in (broken(2, kv_from=2), broken(2, kv_from=1), broken(4, kv_from=2), broken(2, kv_heads=3), broken(2, rot={"dims": 8, "base": 1e3})):
        with pytest.raises(ValueError, match="keys and values"):
            zupupel.config_from_dict(bad)
    with pytest.raises(ValueError, match="rotated part"):
        zupupel.config_from_dict(broken(1, rot={"dims": 4, "base": 300.0}))
    with pytest.raises(ValueError, match="cannot be taken"):
        MoESpec(experts=6, top=4, ff=4, groups=4, keep=1, identity=2)
    for kw in (dict(act="clamped_swish"), dict(limit=1.0), dict(act="clamped_swish", limit=1.0, shared_ff=8)):
        with pytest.raises(ValueError, match="expert activation"):
            MoESpec(experts=6, top=2, ff=4, **kw)
    with pytest.raises(ValueError, match="normed head by head"):
        LayerSpec("attention", heads=1, dim=4, vdim=4, kv_heads=1, qk_norm=True, rot_halves=True)
    for kw in (dict(norm_sum=True, norm_groups=2), dict(sum_alpha=2.0), dict(embed_norm=True, embed_scale=2.0)):
        with pytest.raises(ValueError):
            composed_config("x", [LayerSpec("attention", heads=1, dim=4, vdim=4, kv_heads=1)], 8, 16, **kw)
    with pytest.raises(NotImplementedError, match="rollout engine"):
        GPTModel(get_config("tiny-zupupel"))
    with pytest.raises(NotImplementedError):
        RolloutEngine(get_config("tiny-zupupel"), return_routed_experts=True)
    assert get_config("zupupel-15b").num_parameters() > 1.4e10


def test_column_groups_fit_the_latent_rows():
    from relax_b200.models.config import LayerSpec
    from relax_b200.ops import latent_columns
    from relax_b200.rollout.composed import attention_items, latent_row

    row = lambda rank, rot: (latent_row(LayerSpec("latent_attention", heads=1, dim=8, vdim=8, kv_rank=rank, rot_dims=rot, rot_base=10.0)), (rank + 63) // 64 * 64)
    assert row(20, 6) == (128, 64) and row(512, 64) == (576, 512) and row(64, 0) == (64, 64)
    assert [latent_columns(*row(*x)) for x in ((20, 6), (512, 0), (512, 64), (256, 96))] == [64, 64, 32, 64]
    items = attention_items([3, 40], [10, 90], 20, 32)
    assert all(0 < n <= 32 for _, _, n, _ in items) and sum(n for _, _, n, _ in items) == 43 * 20


def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from relax_b200.entrypoints import trace
    from relax_b200.models import zupupel

    cfg, t = O.random_model(O.CONFIGS["odd"], 9)
    zupupel.save(str(tmp_path / "m"), zupupel.config_from_dict(cfg), t)
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


def test_engine_server_serves_a_zupupel_folder():
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
