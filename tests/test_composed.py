"""Composed stacks (Talizen): reader, loader, cache, scheduler and generation on the CPU against plain float64 statements."""
import io
import json
import os
import sys

import pytest
import torch

sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import composed_driver as D  # noqa: E402
import oracle_composed as O  # noqa: E402

TIGHT = 2e-5


@pytest.mark.parametrize("name", list(O.CONFIGS))
def test_prompt_portions_and_decoding_equal_the_plain_statement(name):
    cfg = O.CONFIGS[name]
    t = O.random_model(cfg, 1, sharp=3.0)
    toks = O.tokens(cfg, 41, 1)
    want = O.model(cfg, t, toks)
    eng = D.engine(cfg, t, blocks=6)
    for sizes in ([41], [1], [2], [16], [17, 1, 3], [2, 15, 1, 1]):
        assert O.distance(D.feed_alone(eng, toks, sizes), want) < TIGHT, sizes
        D.all_free(eng)


def test_unequal_requests_in_one_batch_equal_each_alone_and_slots_and_pages_are_used_again():
    cfg = O.CONFIGS["odd"]
    t = O.random_model(cfg, 2, sharp=4.0)
    seqs = [O.tokens(cfg, n, 10 + n) for n in (33, 5, 48, 2, 17, 20, 31)]
    want = [O.model(cfg, t, s) for s in seqs]
    eng = D.engine(cfg, t, blocks=9)          # fewer pages than all sequences together need
    plans = [[7, 1], [1], [16, 2, 0, 3], [2], [0, 5], [3], [9, 1, 1]]
    got = D.feed_mixed(eng, seqs, plans, [0, 0, 0, 1, 8, 12, 16])
    for g, w in zip(got, want):
        assert O.distance(g, w) < TIGHT
    D.all_free(eng)


def test_state_of_a_freed_slot_does_not_leak():
    cfg = O.CONFIGS["single"]
    t = O.random_model(cfg, 3)
    a, b = O.tokens(cfg, 30, 1), O.tokens(cfg, 9, 2)
    eng = D.engine(cfg, t, blocks=4, state_slots=1)
    D.feed_alone(eng, a, [30])
    assert O.distance(D.feed_alone(eng, b, [4, 1]), O.model(cfg, t, b)) < TIGHT
    r = eng.open_sequence()
    eng.feed([(r, a[:3], [])])
    with pytest.raises(RuntimeError, match="slot"):
        eng.feed([(eng.open_sequence(), b[:2], [])])


def test_steps_without_wanted_logits_and_bad_tokens():
    cfg = O.CONFIGS["single"]
    eng = D.engine(cfg, O.random_model(cfg, 3), blocks=4)
    r = eng.open_sequence()
    assert eng.feed([(r, [1, 2, 3], [])]) is None
    assert eng.feed([(r, [4, 5], [1, 0, 1])]).shape == (3, cfg["vocab"])
    with pytest.raises(ValueError, match="vocabulary"):
        eng.feed([(r, [cfg["vocab"]], [0])])
    with pytest.raises(ValueError, match="at least one token"):
        eng.run_segments([], [])


@pytest.mark.parametrize("windowed", [False, True])
def test_greedy_generation_through_the_scheduler(windowed):
    from relax_b200.rollout.engine import SamplingParams

    cfg = O.CONFIGS["odd"]
    t = O.random_model(cfg, 4, sharp=2.0)
    prompts = [O.tokens(cfg, n, 40 + n) for n in (3, 30, 17, 9, 1)]
    want = [D.greedy(cfg, t, p, 6) for p in prompts]
    # two state slots: requests queue; 11 prompt tokens per step: prompts are cut beside decoding requests
    eng = D.engine(cfg, t, blocks=12, state_slots=2, max_prefill_tokens=11, windowed_decode=windowed, decode_window=3)
    res = eng.generate(prompts, SamplingParams(temperature=0.0, max_new_tokens=6, ignore_eos=True))
    assert [r.output for r in res] == want
    assert all(len(r.logprobs) == 6 and max(r.logprobs) <= 1e-6 for r in res)
    assert eng.sm.num_free == eng.sm.n - 1 and eng.bm.num_free == eng.bm.num_blocks - (1 if windowed else 0)


def test_group_members_share_the_prompt_and_partial_rollouts_resume():
    from relax_b200.rollout.engine import SamplingParams

    cfg = O.CONFIGS["even"]
    t = O.random_model(cfg, 5)
    p = O.tokens(cfg, 37, 3)
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
    eng.add_request(p, SamplingParams(temperature=0.0, max_new_tokens=50, ignore_eos=True))
    for _ in range(5):
        eng.step()
    out = eng.abort_all()
    assert out[0].status == "aborted" and out[0].output[: len(want)] == want[: len(out[0].output)]
    D.all_free(eng)


def test_checkpoint_round_trip_and_registry(tmp_path):
    from relax_b200.checkpoint import hf as H
    from relax_b200.entrypoints.serve import engine_config
    from relax_b200.models import talizen
    from relax_b200.models.config import get_config

    cfg = O.CONFIGS["odd"]
    t = O.random_model(cfg, 6)
    mc = talizen.config_from_dict({"architecture": "Talizen", **cfg})
    assert talizen.config_to_dict(mc) == {"architecture": "Talizen", **cfg}
    assert {k: tuple(v.shape) for k, v in t.items()} == talizen.tensor_shapes(mc)
    assert mc.num_parameters() == sum(v.numel() for v in t.values())
    talizen.save(str(tmp_path), mc, t)
    read = engine_config("tiny", str(tmp_path))
    assert read.layer_specs == mc.layer_specs and read.norm_groups == 3 and read.rms_norm_eps == 3e-5
    H.validate_against_hf(read, str(tmp_path))
    with pytest.raises(ValueError, match="does not match"):
        H.validate_against_hf(get_config("tiny-talizen"), str(tmp_path))
    with pytest.raises(ValueError, match="does not match"):
        H.validate_against_hf(get_config("tiny"), str(tmp_path))
    d = {**talizen.config_to_dict(mc), "architecture": "Nobody"}
    with open(tmp_path / "config.json", "w") as f:
        json.dump(d, f)
    with pytest.raises(ValueError, match="unknown architecture"):
        engine_config("tiny", str(tmp_path))


def test_loader_and_config_reject_what_does_not_fit():
    from relax_b200.models import talizen
    from relax_b200.models.config import LayerSpec, get_config
    from relax_b200.models.transformer import GPTModel
    from relax_b200.rollout.engine import RolloutEngine

    cfg = O.CONFIGS["single"]
    t = O.random_model(cfg, 7)
    for change in ({"l0.mix.extra": torch.zeros(2)}, {"embed": t["embed"][:-1]}):
        with pytest.raises(ValueError, match="does not fit"):
            D.engine(cfg, {**t, **change})
    with pytest.raises(ValueError, match="missing"):
        D.engine(cfg, {k: v for k, v in t.items() if k != "l1.mix.g"})
    with pytest.raises(ValueError, match="unknown mixer type"):
        talizen.config_from_dict({**cfg, "layers": [{**cfg["layers"][0], "type": "gated_conv"}]})
    with pytest.raises(ValueError, match="feed-forward kind"):
        talizen.config_from_dict({**cfg, "layers": [{**cfg["layers"][0], "mlp": {"kind": "routed", "ff": 8}}]})
    with pytest.raises(ValueError, match="groups"):
        talizen.config_from_dict({**cfg, "norm": {"eps": 1e-5, "groups": 5}})
    with pytest.raises(ValueError, match="unknown mixer"):
        LayerSpec("conv", heads=1, dim=1, vdim=1)
    with pytest.raises(NotImplementedError, match="rollout engine"):
        GPTModel(get_config("tiny-talizen"))
    with pytest.raises(NotImplementedError):
        RolloutEngine(get_config("tiny-talizen"), speculative=True)
    with pytest.raises(ValueError, match="empty"):
        from relax_b200.rollout.engine import SamplingParams

        RolloutEngine(get_config("tiny-talizen")).add_request([], SamplingParams())


def test_memory_release_and_flush():
    from relax_b200.rollout.engine import SamplingParams

    cfg = O.CONFIGS["single"]
    t = O.random_model(cfg, 8)
    p = O.tokens(cfg, 12, 1)
    want = D.greedy(cfg, t, p, 3)
    eng = D.engine(cfg, t, blocks=8)
    go = lambda: eng.generate([p], SamplingParams(temperature=0.0, max_new_tokens=3, ignore_eos=True))[0].output
    assert go() == want
    eng.flush_cache()
    eng.release_memory_occupation(("kv_cache",))
    eng.resume_memory_occupation(("kv_cache",))
    assert go() == want


def test_attention_items_cover_every_column_once():
    from relax_b200.rollout.composed import attention_items

    for heads, width in ((5, 64), (16, 64), (64, 64), (70, 64), (130, 64), (1, 16)):
        lens, ctx = [3, 1, 40, 2], [3, 17, 140, 64]
        seen = []
        for seg, c0, n, base in attention_items(lens, ctx, heads, width):
            assert 0 < n <= width
            for c in range(c0, c0 + n):
                row = c // heads
                first = sum(lens[:seg])
                assert first <= row < first + lens[seg]
                assert base + row == ctx[seg] - lens[seg] + (row - first) + 1
            seen += range(c0, c0 + n)
        assert seen == list(range(sum(lens) * heads))


def test_recurrent_spans_cover_every_row_in_whole_chunks():
    from relax_b200.rollout.composed import recurrent_spans

    assert recurrent_spans([5, 1, 100], 2) is None and recurrent_spans([2048] * 4, 32) is None
    for lens, heads in (([8192], 32), ([1, 700, 3, 2049], 16), ([260], 1), ([4000, 4000, 1], 8)):
        spans, first = recurrent_spans(lens, heads, shortest=64)
        row = 0
        for s, n in enumerate(lens):
            part = spans[first[s]:first[s + 1]]
            assert part[0][0] == row and part[-1][1] == row + n
            assert all(a[1] == b[0] and (a[1] - a[0]) % 16 == 0 for a, b in zip(part, part[1:])) and all(b > a for a, b in part)
            row += n
        assert first[-1] == len(spans) > len(lens)


def test_trace_replay_writes_the_wanted_logits(tmp_path):
    from relax_b200.entrypoints import trace
    from relax_b200.models import talizen

    cfg = O.CONFIGS["odd"]
    t = O.random_model(cfg, 9)
    model_dir = tmp_path / "m"
    talizen.save(str(model_dir), talizen.config_from_dict({"architecture": "Talizen", **cfg}), t)
    a, b = O.tokens(cfg, 20, 1), O.tokens(cfg, 6, 2)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:9], "want": [8, 2]}, {"id": "b", "tokens": b[:2], "want": []}], "end": []},
             {"step": 1, "entries": [{"id": "b", "tokens": b[2:], "want": []}], "end": ["b"]},
             {"step": 2, "entries": [{"id": "c", "tokens": b, "want": [5]}, {"id": "a", "tokens": a[9:], "want": [10]}], "end": ["a", "c"]}]
    eng = trace.build_engine(str(model_dir), torch.float32, 128, device="cpu")
    assert eng.bm.num_blocks == 2 and eng.sm.num_free == 4
    done = []
    trace.replay(eng, io.StringIO("".join(json.dumps(s) + "\n" for s in steps)), str(tmp_path), done.append)
    assert done == [0, 1, 2] and not (tmp_path / "1.f32").exists()
    wa, wb = O.model(cfg, t, a), O.model(cfg, t, b)
    for name, rows in (("0", [wa[8], wa[2]]), ("2", [wb[5], wa[19]])):
        got = torch.frombuffer(bytearray((tmp_path / f"{name}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
        assert O.distance(got, torch.stack(rows)) < TIGHT
    D.all_free(eng)


def test_engine_server_serves_a_talizen_folder(tmp_path):
    from relax_b200.models import talizen
    from relax_b200.rollout.engine import SamplingParams
    from relax_b200.rollout.http_server import EngineServer, HTTPEngine

    cfg = O.CONFIGS["single"]
    t = O.random_model(cfg, 10)
    p = O.tokens(cfg, 11, 1)
    eng = D.engine(cfg, t, blocks=16)
    srv = EngineServer(eng)
    try:
        out = HTTPEngine(srv.url).generate([p], SamplingParams(temperature=0.0, max_new_tokens=4, ignore_eos=True))
        assert list(out[0].output) == D.greedy(cfg, t, p, 4)
    finally:
        srv.close() if hasattr(srv, "close") else srv.httpd.shutdown()
    assert talizen.ARCHITECTURE == "Talizen"
