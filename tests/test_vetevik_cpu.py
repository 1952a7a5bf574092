"""Vetevik's host side without a GPU: configuration and registry, weight names, run order, cache needs and
chunked pages, the oracle's own mechanisms, and the whole engine (step function, scheduler) on the stand-in
kernels against the plain implementation."""

from __future__ import annotations

import json
import math

import pytest
import torch

import plain_vetevik as plain
import vetevik_support as vs
from fake_ops import FakeOps
from mini_llm_runtime_b200 import ops
from mini_llm_runtime_b200.cache import CacheManager
from mini_llm_runtime_b200.config import VetevikConfig, config_from_dict, load_config
from mini_llm_runtime_b200.engine import ContinuousBatchEngine
from mini_llm_runtime_b200.models import build_model, write_random_model_dir
from mini_llm_runtime_b200.parts import KVCacheNeed, StateNeed
from mini_llm_runtime_b200.weights.loader import WeightError

F32 = torch.float32
F64 = torch.float64


def test_config_round_trip_and_registry(tmp_path):
    config = config_from_dict(vs.MIXED)
    assert isinstance(config, VetevikConfig) and config.vocab_size == 131 and config.hidden_size == 72
    assert config_from_dict(config.to_dict()) == config and config.to_dict() == vs.MIXED
    assert config_from_dict(vs.PLAIN).to_dict() == vs.PLAIN
    folder = write_random_model_dir(tmp_path / "model", config, seed=3)
    entry, loaded = load_config(folder)
    assert entry.name == "Vetevik" and loaded == config
    stored = json.loads((folder / "config.json").read_text())
    assert stored["loop"] == {"start": 1, "stop": 3, "times": 2} and stored["layers"][2]["mlp"] is None
    # keys that may be left out: kv_heads, vdim of an attention, mask, softcap, norm.groups, residual_mult, loop
    short = {"architecture": "Vetevik", "vocab": 9, "width": 8, "norm": {"eps": 1e-5}, "layers": [
        {"type": "attention", "mixer": {"heads": 2, "dim": 4, "scale": 0.5}, "mlp": None}]}
    small = config_from_dict(short)
    assert (small.norm_groups, small.residual_mult, small.loop_given) == (1, 1.0, False)
    assert small.layers[0].mixer_args == {"heads": 2, "kv_heads": 2, "dim": 4, "scale": 0.5, "softcap": 0.0, "chunk": 0}


@pytest.mark.parametrize("damage,message", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][1]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=8), "vdim"),
    (lambda c: c["layers"][1]["mixer"].update(softcap=-1.0), "softcap"),
    (lambda c: c["layers"][1]["mixer"].update(mask={}), "mask"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=3), "kv_heads"),
    (lambda c: c["layers"][0]["mixer"].update(conv=0), "conv"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][0]["mlp"].pop("expert"), "expert"),
    (lambda c: c["norm"].update(groups=5), "groups"),
    (lambda c: c["loop"].update(stop=9), "loop"),
    (lambda c: c["loop"].pop("times"), "loop"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layer"),
])
def test_config_errors(damage, message):
    data = json.loads(json.dumps(vs.MIXED))
    damage(data)
    with pytest.raises((KeyError, ValueError), match=message):
        config_from_dict(data)


def test_run_order_expected_tensors_and_cache_needs():
    model = build_model(config_from_dict(vs.MIXED), F32)
    steps = model.spec.run_order
    assert [s.layer for s in steps] == [0, 1, 2, 1, 2, 3, 4] and [s.cache for s in steps] == list(range(7))
    assert [s.add_embedding for s in steps] == [False, False, False, True, False, False, False]
    assert [(s.layer, s.add_embedding) for s in build_model(config_from_dict(vs.ODD), F32).spec.run_order] == plain.layer_runs(vs.ODD)
    expected = model.expected_tensors()
    assert expected["embed"].shape == (131, 72) and expected["final.norm"].shape == (72,) and "head" not in expected
    assert expected["l0.mix.q"].shape == (24, 72) and expected["l0.mix.v"].shape == (80, 72) and expected["l0.mix.g"].shape == (80, 72)
    assert expected["l0.mix.k.conv"].shape == (24, 4) and expected["l0.mix.v.conv"].shape == (80, 4)
    assert expected["l0.mix.a"].shape == (4, 72) and expected["l0.mix.norm"].shape == (20,) and expected["l0.mix.o"].shape == (72, 80)
    assert expected["l1.mix.q"].shape == (96, 72) and expected["l1.mix.k"].shape == (32, 72) and "l1.mix.v" not in expected
    assert expected["l1.mix.g"].shape == (96, 72) and expected["l1.mix.sink"].shape == (6,)
    assert expected["l1.norm1b"].shape == (72,) and "l2.norm2" not in expected and "l2.norm2b" not in expected
    assert expected["l0.mlp.router"].shape == (5, 72) and expected["l0.mlp.e4.down"].shape == (72, 24)
    assert "l0.mlp.correction" not in expected
    needs = model.cache_needs()
    assert needs[0] == (StateNeed((4, 20, 12), F32, "state"), StateNeed((3, 128), F32, "conv"))
    assert needs[1] == needs[3] == KVCacheNeed(2, 16, None, value_dim=0, chunk=21)
    assert needs[5] == KVCacheNeed(4, 12, None, value_dim=0, chunk=50)
    tensors = vs.draw_tensors(expected, 1)
    del tensors["l1.mix.sink"]
    tensors["l0.mix.A_log"] = torch.zeros(5, dtype=torch.bfloat16)
    with ops.use(FakeOps()), pytest.raises(WeightError) as error:
        build_model(config_from_dict(vs.MIXED), F32).load(tensors, "cpu")
    assert "l1.mix.sink" in error.value.missing and error.value.wrong_shape[0][0] == "l0.mix.A_log"


def test_what_a_chunked_need_can_see():
    need = KVCacheNeed(1, 8, None, chunk=10)
    assert [need.lowest_visible(p) for p in (0, 9, 10, 19, 25)] == [0, 0, 10, 10, 20] and need.span == 10
    both = KVCacheNeed(1, 8, 4, chunk=10)
    assert [both.lowest_visible(p) for p in (3, 9, 11, 18)] == [0, 6, 10, 15] and both.span == 4
    assert KVCacheNeed(1, 8).span is None and KVCacheNeed(1, 8).lowest_visible(100) == 0


def test_pages_of_chunks_that_have_passed_are_given_back():
    cache = CacheManager([KVCacheNeed(1, 4, None, value_dim=0, chunk=10)], page_size=4, num_pages=8, max_requests=2,
                         max_tokens_per_request=64, dtype=F32, device="cpu", max_step_tokens=6)
    group = cache.groups[0]
    # a request's most pages at once: a chunk but one token, a step, and a page that straddles
    assert cache.pages_for_lifetime(group, 64) == 5 and cache.pages_for_lifetime(group, 8) == 2
    request = cache.create_request("a", lifetime_tokens=64)
    for count, held in ((6, 2), (3, 3), (1, 1), (6, 2), (4, 0), (6, 2)):
        cache.begin_step([("a", count)])
        cache.commit_step()
        assert request.held(0) == held, (request.committed, request.pages)
        first = request.committed // 10 * 10 // 4
        assert all((page < 0) == (logical < first) for logical, page in enumerate(request.pages[0]))
        cache.check_consistency()
    # a step that is taken back gives back only what it took
    before = list(request.pages[0])
    cache.begin_step([("a", 5)])
    cache.abort_step()
    assert request.pages[0] == before
    cache.release("a")
    assert cache.stats().free_pages == (8,)


def test_the_oracles_recurrence_by_hand():
    """One value channel, two key channels: forget, write the gap along the key, read after the write."""
    q = torch.tensor([[1.0, 0.0], [0.5, 2.0]], dtype=F64)
    k = torch.tensor([[1.0, 0.0], [0.6, 0.8]], dtype=F64)
    v = torch.tensor([[3.0], [1.0]], dtype=F64)
    out = plain.delta_recurrence(q, k, v, torch.tensor([0.9, 0.5], dtype=F64), torch.tensor([1.0, 0.25], dtype=F64))
    assert torch.allclose(out[0], torch.tensor([3.0], dtype=F64))            # the state answers the key with its value
    u = 0.25 * (1.0 - 0.6 * 1.5)                                             # the state has faded to (1.5, 0)
    assert torch.allclose(out[1], torch.tensor([0.5 * (1.5 + 0.6 * u) + 2.0 * 0.8 * u], dtype=F64))


def test_the_oracles_attention_by_hand():
    q = torch.ones(5, 1, dtype=F64)
    k = torch.tensor([[0.0], [1.0], [2.0], [-1.0], [0.5]], dtype=F64)
    sink = torch.tensor(0.3, dtype=F64)
    w = plain.attention_weights(q, k, 2.0, 3.0, 0.25, 3, sink)
    bent = 3.0 * torch.tanh(2.0 * k[:, 0] / 3.0)
    first = torch.exp(bent[:3] - 0.25 * torch.tensor([2.0, 1.0, 0.0], dtype=F64))
    assert torch.allclose(w[2, :3], first / (first.sum() + math.exp(0.3))) and float(w[2, 3:].abs().max()) == 0.0
    assert float(w[3, :3].abs().max()) == 0.0 and float(w[3, 3]) > 0.0       # position 3 opens the second chunk
    assert torch.allclose(w[3, 3], torch.exp(bent[3]) / (torch.exp(bent[3]) + math.exp(0.3)))
    assert plain.slopes(4) == [0.25, 0.0625, 0.015625, 0.00390625]


def test_each_mechanism_shows_in_the_oracle():
    """The oracle's answer changes visibly when a mechanism is altered."""
    with ops.use(FakeOps()):
        engine = vs.VEngine(vs.MIXED, F32, "cpu", seed=2)
    tokens = vs.tokens_for(131, 60, 3)
    want = engine.plain(tokens)

    def differs(config_dict=None, tensors=None):
        other = plain.forward(config_dict or vs.MIXED, tensors or engine.tensors, tokens)[0]
        return float((other - want).abs().max()) > 1e-3 * float(want.abs().max())

    def changed(edit):
        data = json.loads(json.dumps(vs.MIXED))
        edit(data)
        return data

    def tensor(name, edit):
        return {**engine.tensors, name: edit(engine.tensors[name].float()).to(torch.bfloat16)}

    assert differs(changed(lambda c: c["loop"].update(times=3)))
    assert differs(changed(lambda c: c["loop"].update(start=2)))
    assert differs(changed(lambda c: c.update(residual_mult=0.7)))
    assert differs(changed(lambda c: c["norm"].update(groups=1)))
    assert differs(changed(lambda c: c["norm"].update(eps=1e-2)))
    assert differs(changed(lambda c: c["layers"][1]["mixer"].update(scale=0.3)))
    assert differs(changed(lambda c: c["layers"][1]["mixer"].update(softcap=3.0)))
    assert differs(changed(lambda c: c["layers"][1]["mixer"].update(mask={"size": 22})))
    assert differs(changed(lambda c: c["layers"][1]["mlp"]["router"].update(top=2)))
    for name in ("l1.mix.sink", "l1.mix.g", "l0.mix.A_log", "l0.mix.dt_bias", "l0.mix.a", "l0.mix.b", "l0.mix.norm", "l0.mix.g",
                 "l2.mix.q.conv", "l0.norm1b", "l0.norm2b", "l0.mlp.router", "final.norm"):
        assert differs(tensors=tensor(name, lambda v: v * 1.5 + 0.25)), name
    assert differs(tensors=tensor("l0.mix.k.conv", lambda v: v.flip(1)))
    # an expert's weight belongs to its input: doubling it is not doubling the output
    t = {f"e.{n}": torch.eye(3, dtype=F64) for n in ("gate", "up", "down")}
    x = torch.tensor([[0.5, -1.0, 2.0]], dtype=F64)
    assert not torch.allclose(plain.expert(2 * x, t, "e."), 2 * plain.expert(x, t, "e."))


def test_state_and_carried_inputs_under_any_cut():
    config = vs.config([vs.delta(2, 1, 8, 6, 4)], width=24, vocab=30)
    with ops.use(FakeOps()):
        engine = vs.VEngine(config, F32, "cpu", seed=5, overrides={"l0.mix.A_log": lambda t: torch.full_like(t, -6.0)})
        tokens = vs.tokens_for(30, 40, 1)
        want = engine.plain(tokens)
        for cuts in ([], [1], [2, 3, 4], [1, 2, 3, 4, 5, 6], range(1, 40), [3, 20, 22]):
            vs.assert_logits_close(engine.run_cuts("r", tokens, cuts), want, F32, f"cuts {list(cuts)[:4]}")


@pytest.mark.parametrize("name", ["MIXED", "ODD", "PLAIN"])
def test_whole_prompt_token_by_token_and_portions(name):
    config = getattr(vs, name)
    with ops.use(FakeOps()):
        engine = vs.VEngine(config, F32, "cpu", seed=1)
        tokens = vs.tokens_for(config["vocab"], 60, 8)
        want = engine.plain(tokens)
        vs.assert_logits_close(engine.run_cuts("whole", tokens, []), want, F32, "whole")
        vs.assert_logits_close(engine.run_cuts("single", tokens, range(1, 60)), want, F32, "token by token")
        vs.assert_logits_close(engine.run_cuts("cut", tokens, [2, 4, 21, 22, 50]), want, F32, "portions")


SMALL = vs.config([vs.delta(2, 1, 8, 12, 3, vs.moe(24, 4, 2)), vs.attention(4, 2, 6, 11), vs.attention(2, 2, 10, 30)],
                  width=40, vocab=70, groups=2, mult=0.8, loop=(0, 2, 2))


def test_batches_pages_and_slots_used_again():
    with ops.use(FakeOps()):
        engine = vs.VEngine(SMALL, F32, "cpu", seed=3, page_size=8, num_pages=[8, 14], max_requests=2, max_tokens=64,
                            max_step_tokens=16)
        for number in range(3):
            prompts = {f"a{number}": vs.tokens_for(70, 33 + 7 * number, 20 + number),
                       f"b{number}": vs.tokens_for(70, 25, 30 + number)}
            plan = []
            for start in range(0, 60, 6):
                step = {name: min(6, len(tokens) - start) for name, tokens in prompts.items() if start < len(tokens)}
                if step:
                    plan.append(step)
            got = engine.run_plan(prompts, plan)
            for name, tokens in prompts.items():
                vs.assert_logits_close(got[name], engine.plain(tokens), F32, name)
            engine.cache.check_consistency()
        assert engine.cache.stats().free_pages == (8, 14) and engine.cache.stats().free_slots == 2


def test_greedy_generation_through_the_scheduler():
    with ops.use(FakeOps()):
        parts = vs.VEngine(vs.MIXED, F32, "cpu", seed=31)
        engine = ContinuousBatchEngine.from_model(parts.model, block_size=8, total_blocks=96, max_running_requests=3,
                                                  max_batch_tokens=24, max_model_len=120)
        prompts = [vs.tokens_for(131, length, 40 + i) for i, length in enumerate([5, 37, 18, 2])]
        generated = engine.generate(prompts, max_new_tokens=6)
    for prompt, got in zip(prompts, generated):
        sequence = list(prompt)
        for _ in range(6):
            sequence.append(int(torch.argmax(parts.plain(sequence)[-1])))
        assert got == sequence[len(prompt):]


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random(seed):
    config = vs.random_config(seed)
    with ops.use(FakeOps()):
        engine = vs.VEngine(config, F32, "cpu", seed=seed, num_pages=40)
        prompts = {"a": vs.tokens_for(config["vocab"], 45, seed), "b": vs.tokens_for(config["vocab"], 21, seed + 50)}
        got = engine.run_plan(prompts, [{"a": 17, "b": 1}, {"a": 1, "b": 2}, {"a": 2, "b": 18}, {"a": 25}])
    for name, tokens in prompts.items():
        vs.assert_logits_close(got[name], engine.plain(tokens), F32, f"seed {seed} {name}")
