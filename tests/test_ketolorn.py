"""Ketolorn stacks: every mechanism, the reader, cache, scheduler and generation on the CPU against plain float64 statements."""
import io
import json
import math
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import composed_driver as D  # noqa: E402
import oracle_ketolorn as O  # noqa: E402
from oracle_composed import distance, tokens  # noqa: E402

F64 = torch.float64
TIGHT = 2e-5


def _close(got, want, tol):
    err = (got.to(F64) - want.to(F64)).abs().max().item()
    assert err <= tol * max(1.0, want.abs().max().item()), (err, want.abs().max().item())


# ---------------------------------------------------------------------------------------------------- mechanisms alone


@pytest.mark.parametrize("dim,vdim,rot,norm", [(18, 13, 10, True), (16, 16, 16, True), (12, 20, 4, False), (7, 5, 0, True)])
def test_turned_and_normed_heads_go_to_their_pages(dim, vdim, rot, norm):
    from relax_b200 import ops

    H, G, T, eps = 6, 2, 5, 1e-3
    g = torch.Generator().manual_seed(dim)
    x = torch.randn(T, H * dim + G * (dim + vdim) + 3, generator=g)
    pos = torch.tensor([0, 1, 77, 1500, 30000], dtype=torch.int32)
    freq = torch.tensor([50.0 ** (-2 * i / max(rot, 1)) for i in range(rot // 2)], dtype=F64)
    kp, vp = torch.zeros(40, G, 32), torch.zeros(40, G, 32)
    slots = torch.tensor([3, 39, 0, 17, 16])
    table = ops.rope_table(pos + 2, -2, freq) if rot else None
    q = ops.attention_inputs(x, table, H, G, dim, vdim, 32, rot, eps if norm else 0.0, kp, vp, slots)
    for got, a, n in ((q, 0, H), (kp[slots], H * dim, G)):
        want = O.turn(x[:, a:a + n * dim].to(F64).view(T, n, dim), pos.tolist(), rot, 50.0)
        _close(got[..., :dim], O.rms(want, eps) if norm else want, 2e-6)
        assert not got[..., dim:].any()
    _close(vp[slots, :, :vdim], x[:, (H + G) * dim:(H + G) * dim + G * vdim].view(T, G, vdim), 0)
    only_q = ops.attention_inputs(x[:, : H * dim], table, H, G, dim, vdim, 32, rot, eps if norm else 0.0, None, None, slots)
    assert torch.equal(only_q, q)


def _pools(lens, G, dim, vdim, page, seed):
    g = torch.Generator().manual_seed(seed)
    nb = [-(-L // page) for L in lens]
    perm = torch.randperm(sum(nb) + 2, generator=g).tolist()
    bt = torch.zeros(len(lens), max(nb) + 1, dtype=torch.int32)
    for s, n in enumerate(nb):
        bt[s, :n] = torch.tensor([perm.pop() for _ in range(n)])
    rows = [torch.tensor([int(bt[s, p // page]) * page + p % page for p in range(L)]) for s, L in enumerate(lens)]
    return torch.randn((sum(nb) + 2) * page, G, dim, generator=g), torch.randn((sum(nb) + 2) * page, G, vdim, generator=g), bt, rows


@pytest.mark.parametrize("sink", [None, 2.0, 40.0, -60.0])
def test_attention_over_pages_with_a_sink(sink):
    from relax_b200.ops import reference as ref

    H, G, dim, vdim, page, scale = 6, 2, 10, 7, 4, 0.8
    lens, ctx = [1, 3, 6], [5, 9, 6]
    k, v, bt, rows = _pools(ctx, G, dim, vdim, page, 3)
    q = torch.randn(10, H, dim, generator=torch.Generator().manual_seed(1))
    sk = None if sink is None else sink + torch.randn(H, generator=torch.Generator().manual_seed(2))
    got = ref.paged_attention(q, k, v, bt, page, torch.tensor(ctx), torch.tensor([0, 1, 4, 10]), scale, sk, 8).view(10, H, 8)
    at = 0
    for s, (n, L) in enumerate(zip(lens, ctx)):
        want = O.attend(q[at:at + n].to(F64), k[rows[s]].to(F64), v[rows[s]].to(F64), L - n, scale, None if sk is None else sk.to(F64))
        _close(got[at:at + n, :, :vdim], want, 1e-5)
        at += n
    assert not got[..., vdim:].any()


@pytest.mark.parametrize("E,top,groups,keep", [(15, 4, 5, 3), (8, 8, 4, 4), (6, 1, 6, 1), (10, 4, 2, 1), (9, 2, 1, 1)])
def test_router_keeps_groups_and_weights_by_scores(E, top, groups, keep):
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    spec = MoESpec(experts=E, top=top, ff=8, groups=groups, keep=keep)
    z = torch.randn(60, E + 4, generator=torch.Generator().manual_seed(E)) * 2
    z[0, :E], z[1, :E] = -30.0 - torch.arange(E), 12.0 - torch.arange(E)
    plan = ops.moe_route(z, spec, torch.float32)
    for t in range(60):
        s = (1 / (1 + torch.exp(-z[t, :E].to(F64)))).tolist()
        chosen, gap = O.choose(s, top, groups, keep)
        if gap > 1e-6:
            assert plan.index[t].tolist() == chosen
            assert all(abs(a - s[e]) < 1e-6 for a, e in zip(plan.weight[t].tolist(), chosen))


def test_group_rule_decides_against_the_best_single_expert():
    """Two good experts of one group beat the best expert of another."""
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    z = torch.tensor([[4.0, -9.0, 2.0, 2.1], [4.0, 1.0, 0.9, 0.8]])
    plan = ops.moe_route(z, MoESpec(experts=4, top=1, ff=8, groups=2, keep=1), torch.float32)
    assert plan.index.tolist() == [[3], [0]]
    plan = ops.moe_route(z, MoESpec(experts=4, top=2, ff=8, groups=2, keep=1, renormalize=True, weight_scale=3.0), torch.float32)
    assert torch.allclose(plan.weight.sum(1), torch.tensor([3.0, 3.0]))


def test_experts_and_shared_expert_join_before_the_norm():
    from relax_b200 import ops
    from relax_b200.models.config import MoESpec

    g = torch.Generator().manual_seed(5)
    n = lambda *s: torch.randn(*s, generator=g)
    W, E, ff, T, spec = 24, 6, 10, 9, MoESpec(experts=6, top=2, ff=10, groups=3, keep=2, shared_ff=14)
    h, router, up, down, su, sd = n(T, W), n(E, W), n(E, ff, W), n(E, W, ff), n(14, W), n(W, 14)
    w = {"router": router, "shared.up": su, "shared.down": sd, **{f"e{e}.up": up[e] for e in range(E)}, **{f"e{e}.down": down[e] for e in range(E)}}
    want, _ = O.routed(h.to(F64), {k: x.to(F64) for k, x in w.items()},
                       {"router": {"top": 2, "groups": {"count": 3, "keep": 2}}, "shared": {}})
    plan = ops.moe_route(ops.linear_fp32(h, router), spec, torch.float32)
    rows = ops.moe_experts(h, plan, up, down, "relu2")
    res, nw = n(T, W), n(W)
    total = res.to(F64) + O.rms(want, 1e-4) * nw.to(F64)
    out = ops.norm_add(res, ops.linear(ops.linear_act(h, su, "relu2"), sd), nw, W, 1, 1e-4, None, (rows, plan))
    _close(out, total, 1e-5)
    assert out.data_ptr() != 0 and torch.equal(out, res)


def test_embedded_tokens_are_normed():
    from relax_b200 import ops

    g = torch.Generator().manual_seed(6)
    table, w = torch.randn(9, 16, generator=g), torch.randn(16, generator=g)
    table[:, 12:], w[12:] = 0, 0
    res, h = ops.embed_rows(torch.tensor([3, 8]), table, w, 12, 1, 1e-2)
    _close(res[:, :12], O.rms(table[[3, 8], :12].to(F64), 1e-2) * w[:12].to(F64), 1e-6)
    assert torch.equal(res, h) and not res[:, 12:].any()


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
    toks = tokens(cfg, 30, 1)
    want = O.model(cfg, t, toks)

    def changed(**tensors):
        return distance(O.model(cfg, {**t, **tensors}, toks), want)

    assert changed(**{"l2.mix.sink": torch.full((6,), -1e9)}) > 1e-2                       # no sink
    assert changed(**{"l0.mix.sink": t["l0.mix.sink"] * 0.31}) > 1e-3                      # sink scaled like a score
    assert changed(**{"embed.norm": torch.ones(cfg["width"])}) > 1e-2
    for path, value in ((("rot", "base"), 1.1e3), (("scale",), 0.3), (("rot", "dims"), 8)):
        other = json.loads(json.dumps(cfg))
        m = other["layers"][0]["mixer"]
        for k in path[:-1]:
            m = m[k]
        m[path[-1]] = value
        assert distance(O.model(other, t, toks), want) > 1e-3, path
    other = json.loads(json.dumps(cfg))
    other["layers"][4]["mixer"]["kv_from"] = 0
    other["layers"][3]["mlp"]["router"]["groups"] = {"count": 1, "keep": 1}
    assert distance(O.model(other, t, toks), want) > 1e-2                                  # groups ignored
    last = lambda n: O.model(cfg, t, toks[:n] + [(toks[n] + 1) % cfg["vocab"]] + toks[n + 1:])[-1:]
    assert all(distance(last(n), want[-1:]) > 1e-3 for n in (0, 1, 15, 16, 28))            # every key counts


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


def test_readers_share_one_pair_of_pools():
    cfg, t = O.random_model(O.CONFIGS["odd"], 2)
    eng = D.engine(cfg, t, blocks=4)
    kv = eng.kv.kv
    assert kv[2][0] is kv[0][0] and kv[4][1] is kv[0][1] and kv[3][0] is kv[1][0] and kv[0][0] is not kv[1][0] and len(eng.kv.paged) == 4


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

    cfg, t = O.random_model(O.CONFIGS["even"], 5)
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


def test_checkpoint_round_trip_and_registry(tmp_path):
    from relax_b200.checkpoint import hf as H
    from relax_b200.entrypoints.serve import engine_config
    from relax_b200.models import ketolorn
    from relax_b200.models.config import get_config

    cfg, t = O.random_model(O.CONFIGS["odd"], 6)
    mc = ketolorn.config_from_dict(cfg)
    assert ketolorn.config_to_dict(mc) == cfg
    assert {k: tuple(v.shape) for k, v in t.items()} == ketolorn.tensor_shapes(mc)
    assert mc.num_parameters() == sum(v.numel() for v in t.values())
    ketolorn.save(str(tmp_path), mc, t)
    read = engine_config("tiny", str(tmp_path))
    assert read.layer_specs == mc.layer_specs and read.embed_norm and read.tie_word_embeddings and read.rms_norm_eps == 3e-5
    H.validate_against_hf(read, str(tmp_path))
    with pytest.raises(ValueError, match="does not match"):
        H.validate_against_hf(get_config("tiny-ketolorn"), str(tmp_path))
    eng = D.engine(cfg, t, blocks=4)
    H.load_hf_into_rollout(str(tmp_path), read, eng.weights)
    toks = tokens(cfg, 9, 1)
    assert distance(D.feed_alone(eng, toks, [9]), O.model(cfg, t, toks)) < TIGHT


def test_loader_and_config_reject_what_does_not_fit():
    from relax_b200.models import ketolorn
    from relax_b200.models.config import LayerSpec, MoESpec, get_config
    from relax_b200.models.transformer import GPTModel
    from relax_b200.rollout.engine import RolloutEngine

    cfg, t = O.random_model(O.CONFIGS["odd"], 7)
    for change in ({"l0.mix.extra": torch.zeros(2)}, {"embed": t["embed"][:-1]}, {"l2.mix.k": t["l0.mix.k"]}):
        with pytest.raises(ValueError, match="does not fit"):
            D.engine(cfg, {**t, **change})
    with pytest.raises(ValueError, match="missing"):
        D.engine(cfg, {k: v for k, v in t.items() if k != "l1.mix.sink"})

    def broken(layer, **mixer):
        c = json.loads(json.dumps(cfg))
        c["layers"][layer]["mixer"].update(mixer)
        return c

    with pytest.raises(ValueError, match="unknown mixer type"):
        ketolorn.config_from_dict({**cfg, "layers": [{**cfg["layers"][0], "type": "conv"}]})
    with pytest.raises(ValueError, match="feed-forward kind"):
        ketolorn.config_from_dict({**cfg, "layers": [{**cfg["layers"][0], "mlp": {"kind": "mixture", "ff": 8}}]})
    for bad in (broken(2, kv_from=2), broken(2, kv_from=3), broken(4, kv_from=2), broken(2, kv_heads=3), broken(2, rot={"dims": 8, "base": 1e3})):
        with pytest.raises(ValueError, match="keys and values"):
            ketolorn.config_from_dict(bad)
    with pytest.raises(ValueError, match="do not divide"):
        ketolorn.config_from_dict(broken(0, kv_heads=4))
    with pytest.raises(ValueError, match="bad rotation"):
        LayerSpec("attention", heads=1, dim=4, vdim=4, kv_heads=1, rot_dims=6, rot_base=10.0)
    with pytest.raises(ValueError, match="cannot be taken"):
        MoESpec(experts=8, top=3, ff=4, groups=4, keep=1)
    with pytest.raises(NotImplementedError, match="rollout engine"):
        GPTModel(get_config("tiny-ketolorn"))
    with pytest.raises(NotImplementedError):
        RolloutEngine(get_config("tiny-ketolorn"), return_routed_experts=True)
    assert get_config("ketolorn-16b").num_parameters() > 1.2e10


def test_query_tiles_cover_every_row_once():
    from relax_b200.rollout.composed import query_blocks, tile_tokens
    from relax_b200.models.config import LayerSpec

    spec = lambda H, G: LayerSpec("attention", heads=H, dim=8, vdim=8, kv_heads=G)
    assert [tile_tokens(spec(H, G)) for H, G in ((8, 8), (8, 1), (6, 2), (300, 1))] == [128, 16, 42, 1]
    lens, ctx = [3, 1, 40, 17], [3, 17, 140, 64]
    tiles = query_blocks(lens, ctx, 16)
    assert [-(b[2] + b[3]) for b in tiles] == sorted(-(b[2] + b[3]) for b in tiles)
    seen = []
    for seg, row, n, pos in tiles:
        first = sum(lens[:seg])
        assert 0 < n <= 16 and first <= row and row + n <= first + lens[seg] and pos == ctx[seg] - lens[seg] + row - first
        seen += range(row, row + n)
    assert sorted(seen) == list(range(sum(lens)))


def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from relax_b200.entrypoints import trace
    from relax_b200.models import ketolorn

    cfg, t = O.random_model(O.CONFIGS["odd"], 9)
    ketolorn.save(str(tmp_path / "m"), ketolorn.config_from_dict(cfg), t)
    a, b = tokens(cfg, 20, 1), tokens(cfg, 6, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:9], "want": [8, 2]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": b, "want": [5]}, {"id": "a", "tokens": a[9:], "want": [10]}], "end": ["a", "c"]}]
    eng = trace.build_engine(str(tmp_path / "m"), torch.float32, 128, device="cpu")
    assert eng.bm.num_blocks == 2 and eng.sm.num_free == 4
    done = []
    trace.replay(eng, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), done.append)
    assert done == [0, 1, 2] and not (tmp_path / "1.f32").exists()
    wa, wb = O.model(cfg, t, a), O.model(cfg, t, b)
    for name, rows in (("0", [wa[8], wa[2]]), ("2", [wb[5], wa[19]])):
        got = torch.frombuffer(bytearray((tmp_path / f"{name}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert distance(got, torch.stack(rows)) < TIGHT
    D.all_free(eng)


def test_engine_server_serves_a_ketolorn_folder():
    from relax_b200.rollout.engine import SamplingParams
    from relax_b200.rollout.http_server import EngineServer, HTTPEngine

    cfg, t = O.random_model(O.CONFIGS["single"], 10)
    p = tokens(cfg, 11, 1)
    eng = D.engine(cfg, t, blocks=16)
    srv = EngineServer(eng)
    try:
        out = HTTPEngine(srv.url).generate([p], SamplingParams(temperature=0.0, max_new_tokens=4, ignore_eos=True))
        assert list(out[0].output) == D.greedy(cfg, t, p, 4)
    finally:
        srv.close() if hasattr(srv, "close") else srv.httpd.shutdown()
    assert math.isfinite(out[0].logprobs[0])
