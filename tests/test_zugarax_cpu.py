"""Zugarax's host side without a GPU: configuration and registry, weight names, run order and cache needs, frequency
scalings, the oracle's own mechanisms, and the whole engine (step function, scheduler) on the stand-in kernels against
the plain implementation."""

from __future__ import annotations

import json
import math

import pytest
import torch

import plain_zugarax as plain
import zugarax_support as zs
from fake_ops import FakeOps
from mini_llm_runtime_b200 import ops
from mini_llm_runtime_b200.config import PartSpec, ZugaraxConfig, config_from_dict, load_config
from mini_llm_runtime_b200.engine import ContinuousBatchEngine
from mini_llm_runtime_b200.models import build_model, write_random_model_dir
from mini_llm_runtime_b200.parts import KVCacheNeed, StateNeed, build_part
from mini_llm_runtime_b200.weights.loader import WeightError

F32 = torch.float32
F64 = torch.float64


def test_config_round_trip_and_registry(tmp_path):
    config = config_from_dict(zs.MIXED)
    assert isinstance(config, ZugaraxConfig) and config.vocab_size == 131 and config.hidden_size == 72
    assert config_from_dict(config.to_dict()) == config and config.to_dict() == zs.MIXED
    assert config_from_dict(zs.PLAIN).to_dict() == zs.PLAIN
    folder = write_random_model_dir(tmp_path / "model", config, seed=3)
    entry, loaded = load_config(folder)
    assert entry.name == "Zugarax" and loaded == config
    stored = json.loads((folder / "config.json").read_text())
    assert stored["layers"][3]["mixer"]["kv_from"] == 1 and stored["layers"][3]["mlp"] is None
    # keys that may be left out: kv_heads and vdim of an attention, rot.dims, rot.scaling, embedding, logit_softcap
    short = {"architecture": "Zugarax", "vocab": 9, "width": 8, "norm": {"eps": 1e-5}, "layers": [
        {"type": "attention", "mixer": {"heads": 2, "dim": 4, "scale": 0.5, "mask": {"size": 3}, "rot": {"base": 10.0}}}]}
    small = config_from_dict(short)
    assert (small.embedding_scale, small.logit_softcap) == (1.0, 0.0)
    args = small.layers[0].mixer_args
    assert (args["kv_heads"], args["vdim"], args["rot_dims"], args["rot_scaling"], args["window"]) == (2, 4, 4, (), 3)


@pytest.mark.parametrize("damage,message", [
    (lambda c: c["layers"][0].update(type="conv"), "type"),
    (lambda c: c["layers"][2]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][2]["mixer"].pop("mask"), "mask"),
    (lambda c: c["layers"][2]["mixer"]["mask"].update(size=0), "mask.size"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=4), "kv_heads"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=22), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=5), "rot.dims"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("high"), "scaling"),
    (lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].pop("slow"), "scaling"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=5), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=2), "kv_from"),
    (lambda c: c["layers"][6]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_rank=32), "kv_rank"),
    (lambda c: c["layers"][3]["mixer"]["rot"].update(base=5.0), "rotation"),
    (lambda c: c["layers"][0]["mixer"].update(gate_cap=0), "gate_cap"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "kind"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c.update(logit_softcap=-1.0), "logit_softcap"),
    (lambda c: c.pop("norm"), "norm"),
    (lambda c: c.update(layers=[]), "layer"),
])
def test_config_errors(damage, message):
    data = json.loads(json.dumps(zs.MIXED))
    damage(data)
    with pytest.raises((KeyError, ValueError), match=message):
        config_from_dict(data)


def test_run_order_expected_tensors_and_cache_needs():
    model = build_model(config_from_dict(zs.MIXED), F32)
    steps = model.spec.run_order
    assert [s.layer for s in steps] == list(range(8))
    assert [s.cache for s in steps] == [0, 1, 2, 1, 3, 4, 1, 5]
    assert [s.writes_cache for s in steps] == [True, True, True, False, True, True, False, True]
    expected = model.expected_tensors()
    assert expected["embed"].shape == (131, 72) and expected["head"].shape == (131, 72) and expected["final.norm"].shape == (72,)
    assert expected["l0.mix.q"].shape == (36, 72) and expected["l0.mix.v"].shape == (60, 72) and expected["l0.mix.g"].shape == (60, 72)
    assert expected["l0.mix.i"].shape == (3, 72) and expected["l0.mix.f.b"].shape == (3,) and expected["l0.mix.norm"].shape == (60,)
    assert expected["l1.mix.q"].shape == (96, 72) and expected["l1.mix.dkv"].shape == (48, 72) and expected["l1.mix.uk"].shape == (64, 40)
    assert "l3.mix.dkv" not in expected and "l3.mix.dkv.norm" not in expected and expected["l3.mix.uv"].shape == (24, 40)
    assert "l1.mix.g" not in expected and "l1.mix.dq" not in expected
    assert expected["l2.mix.v"].shape == (56, 72) and expected["l2.mix.g"].shape == (168, 72) and expected["l2.mix.k.norm"].shape == (20,)
    assert "l2.mix.sink" not in expected and "l3.norm2" not in expected
    assert expected["l0.mlp.gate.b"].shape == (56,) and expected["l0.mlp.down.b"].shape == (72,)
    needs = model.cache_needs()
    assert needs[0] == (StateNeed((3, 21, 12), F32, "state"), StateNeed((3,), F32, "maximum"))
    assert needs[1] == KVCacheNeed(1, 48, None, value_dim=0) and needs[2] == KVCacheNeed(2, 20, 21, value_dim=28)
    assert needs[5] == KVCacheNeed(3, 16, 50)
    tensors = zs.draw_tensors(expected, 1)
    del tensors["l2.mix.q.norm"]
    tensors["l0.mix.i.b"] = torch.zeros(5, dtype=torch.bfloat16)
    with ops.use(FakeOps()), pytest.raises(WeightError) as error:
        build_model(config_from_dict(zs.MIXED), F32).load(tensors, "cpu")
    assert "l2.mix.q.norm" in error.value.missing and error.value.wrong_shape[0][0] == "l0.mix.i.b"


@pytest.mark.parametrize("dims,base,scaling", [
    (32, 20000.0, zs.bands(4.0, 1.0, 5.0, 600)), (12, 90.0, zs.bands(5.0, 1.5, 6.0, 48)), (2, 30.0, zs.bands(2.0, 1.0, 4.0, 100)),
    (64, 5e5, zs.bands(8.0, 1.0, 4.0, 8192)), (16, 1e4, None)])
def test_banded_frequencies(dims, base, scaling):
    spec = PartSpec("rope_pairs", {"head_dim": dims, "theta": base, "scaling": {} if scaling is None else {"kind": "bands", **scaling}})
    part = build_part("position", spec, F32)
    part.load({}, torch.device("cpu"))
    want = torch.tensor(plain.banded_frequencies(dims, zs.rotation(base, dims, scaling)), dtype=F64)
    assert torch.allclose(part.rotary_frequencies().double(), want, rtol=1e-6, atol=0) and part.magnitude == 1.0
    if scaling is not None and dims == 32:      # short wavelengths as they are, long ones stretched, some in between
        plainly = torch.tensor(plain.plain_frequencies(dims, base), dtype=F64)
        ratio = want / plainly
        assert float(ratio.max()) == 1.0 and float(ratio.min()) == 0.25 and bool(((ratio > 0.26) & (ratio < 0.99)).any())


@pytest.mark.parametrize("dims,base,scaling", [(24, 90000.0, zs.ramp(6.0, 2000, 20.0, 1.0)), (8, 700.0, zs.ramp(3.0, 60, 6.0, 1.5)),
                                               (6, 77.0, zs.ramp(2.0, 40, 8.0, 1.0)), (2, 10.0, zs.ramp(5.0, 9, 3.0, 1.0))])
def test_ramped_frequencies_and_their_magnitude(dims, base, scaling):
    part = build_part("position", PartSpec("rope_pairs", {"head_dim": dims, "theta": base, "layout": "interleaved",
                                                          "scaling": {"kind": "ramp", **scaling}}), F32)
    part.load({}, torch.device("cpu"))
    want, magnitude = plain.ramped_frequencies(dims, zs.rotation(base, dims, scaling))
    assert torch.allclose(part.rotary_frequencies().double(), torch.tensor(want, dtype=F64), rtol=1e-6, atol=0)
    assert part.magnitude == pytest.approx(magnitude) and part.interleaved


def test_unknown_choices_are_refused():
    with pytest.raises(ValueError, match="scaling"):
        build_part("position", PartSpec("rope_pairs", {"head_dim": 8, "theta": 10.0, "scaling": {"kind": "steps", "factor": 2.0}}), F32)
    with pytest.raises(ValueError, match="sink"):
        build_part("mixer", PartSpec("shaped_attention", {"hidden_size": 8, "heads": 2, "dim": 4, "scale": 1.0, "sink": "other"}), F32)
    with pytest.raises(ValueError, match="biases"):
        build_part("feed_forward", PartSpec("gated_mlp", {"hidden_size": 8, "intermediate_size": 8, "bias": True}), F32)


def test_the_oracles_memory_by_hand():
    """One key channel, one value channel: the gates' exponentials, the running maximum that starts at zero, and the two
    branches of the normaliser."""
    q, k, v = (torch.tensor(x, dtype=F64).view(-1, 1) for x in ([1.0, 2.0], [0.5, 1.0], [3.0, -1.0]))
    log_in, log_forget = torch.tensor([-2.0, 1.0], dtype=F64), torch.tensor([-0.5, -0.25], dtype=F64)
    out = plain.matrix_memory(q, k, v, log_in, log_forget)
    # in absolute terms: n_1 = e^-2 / 2 (below one, so the guard e^-m against e^-m n decides), S_1 = 3 n_1
    n1 = math.exp(-2.0) * 0.5
    assert math.isclose(float(out[0]), 3.0 * n1 / (1.0 + 1e-6 * math.exp(-0.5)), rel_tol=1e-9)      # m_1 = -0.5
    n2, s2 = math.exp(-0.25) * n1 + math.e, math.exp(-0.25) * 3.0 * n1 - math.e
    assert math.isclose(float(out[1]), s2 * 2.0 / (n2 * 2.0 + 1e-6 * math.e), rel_tol=1e-9)          # m_2 = 1, |n q| > 1


def test_the_oracles_window_by_hand():
    q = torch.ones(5, 1, dtype=F64)
    k = torch.tensor([[0.0], [1.0], [2.0], [-1.0], [0.5]], dtype=F64)
    w = plain.window_weights(q, k, 2.0, 3)
    e = torch.exp(2.0 * k[:, 0])
    assert torch.allclose(w[0, 0], e[0] / (1 + e[0])) and torch.allclose(w[4, 2:], e[2:] / (1 + e[2:].sum()))
    assert float(w[4, :2].abs().max()) == 0.0 and float(w[3, 0]) == 0.0 and float(w[3, 1]) > 0.0


def test_each_mechanism_shows_in_the_oracle():
    """The oracle's answer changes visibly when a mechanism is altered."""
    with ops.use(FakeOps()):
        engine = zs.ZuEngine(zs.MIXED, F32, "cpu", seed=2)
    tokens = zs.tokens_for(131, 60, 3)
    want = engine.plain(tokens)

    def differs(config_dict=None, tensors=None):
        other = plain.forward(config_dict or zs.MIXED, tensors or engine.tensors, tokens)[0]
        return float((other - want).abs().max()) > 1e-3 * float(want.abs().max())

    def changed(edit):
        data = json.loads(json.dumps(zs.MIXED))
        edit(data)
        return data

    def tensor(name, edit):
        return {**engine.tensors, name: edit(engine.tensors[name].float()).to(torch.bfloat16)}

    assert differs(changed(lambda c: c["embedding"].update(scale=2.0)))
    assert differs(changed(lambda c: c.update(logit_softcap=9.0)))
    assert differs(changed(lambda c: c["norm"].update(eps=1e-1)))
    assert differs(changed(lambda c: c["layers"][2]["mixer"].update(scale=0.3)))
    assert differs(changed(lambda c: c["layers"][2]["mixer"].update(mask={"size": 22})))
    assert differs(changed(lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10)))
    assert differs(changed(lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].update(factor=4.0)))
    assert differs(changed(lambda c: c["layers"][1]["mixer"]["rot"]["scaling"].update(factor=2.0)))
    assert differs(changed(lambda c: c["layers"][1]["mixer"].update(scale=0.1)))
    assert differs(changed(lambda c: c["layers"][0]["mixer"].update(gate_cap=3.0)))
    assert differs(changed(lambda c: c["layers"][2]["mlp"].update(limit=0.7)))
    for name in ("l2.mix.g", "l2.mix.q.norm", "l2.mix.k.norm", "l1.mix.dkv.norm", "l3.mix.uk", "l6.mix.uv", "l0.mix.i.b", "l0.mix.f.b",
                 "l0.mix.norm", "l0.mix.g", "l0.mlp.gate.b", "l0.mlp.up.b", "l0.mlp.down.b", "l0.norm1", "l0.norm2", "final.norm", "head"):
        assert differs(tensors=tensor(name, lambda v: v * 1.5 + 0.25)), name


def test_a_shared_latent_is_the_first_layers():
    """The reading layer uses what the first one cached: a change of the first layer's latent weights shows in a model
    whose first layer adds nothing to the stream."""
    config, overrides = zs.dominant_latent_case(40, 30, 3, seed=1, shared=True)
    tokens = list(range(40))
    with ops.use(FakeOps()):
        engine = zs.ZuEngine(config, F32, "cpu", seed=5, overrides=overrides)
        want = engine.plain(tokens)
        zs.assert_logits_close(engine.run_cuts("a", tokens, [2, 17, 30, 31]), want, F32)
        assert engine.cache.stats().free_pages == (64,)      # one group, one entry: the second layer keeps nothing
    other = dict(engine.tensors)
    other["l0.mix.dkv"] = other["l0.mix.dkv"].roll(1, 0)
    assert float((engine.plain(tokens, tensors=other) - want).abs().max()) > 0.1


def test_state_under_any_cut():
    config = zs.config([zs.mlstm(2, 8, 6, 10.0)], width=24, vocab=30)
    with ops.use(FakeOps()):
        engine = zs.ZuEngine(config, F32, "cpu", seed=5, overrides={"l0.mix.f.b": lambda t: torch.full_like(t, 6.0)})
        tokens = zs.tokens_for(30, 40, 1)
        want = engine.plain(tokens)
        for cuts in ([], [1], [2, 3, 4], [1, 2, 3, 4, 5, 6], range(1, 40), [3, 20, 22]):
            zs.assert_logits_close(engine.run_cuts("r", tokens, cuts), want, F32, f"cuts {list(cuts)[:4]}")


@pytest.mark.parametrize("name", ["MIXED", "ODD", "PLAIN"])
def test_whole_prompt_token_by_token_and_portions(name):
    config = getattr(zs, name)
    with ops.use(FakeOps()):
        engine = zs.ZuEngine(config, F32, "cpu", seed=1)
        tokens = zs.tokens_for(config["vocab"], 60, 8)
        want = engine.plain(tokens)
        zs.assert_logits_close(engine.run_cuts("whole", tokens, []), want, F32, "whole")
        zs.assert_logits_close(engine.run_cuts("single", tokens, range(1, 60)), want, F32, "token by token")
        zs.assert_logits_close(engine.run_cuts("cut", tokens, [2, 4, 21, 22, 50]), want, F32, "portions")


SMALL = zs.config([zs.latent(2, 8, 4, 6, 12), zs.mlstm(2, 8, 12, 8.0, zs.dense(24, 1.0)),
                   zs.attention(4, 2, 6, 10, 11, zs.rotation(100.0, 4)), zs.latent(3, 6, 4, 8, 12, kv_from=0)], width=40, vocab=70)


def test_batches_pages_and_slots_used_again():
    with ops.use(FakeOps()):
        engine = zs.ZuEngine(SMALL, F32, "cpu", seed=3, page_size=8, num_pages=[14, 8], max_requests=2, max_tokens=64,
                             max_step_tokens=16)
        for number in range(3):
            prompts = {f"a{number}": zs.tokens_for(70, 33 + 7 * number, 20 + number),
                       f"b{number}": zs.tokens_for(70, 25, 30 + number)}
            plan = []
            for start in range(0, 60, 6):
                step = {name: min(6, len(tokens) - start) for name, tokens in prompts.items() if start < len(tokens)}
                if step:
                    plan.append(step)
            got = engine.run_plan(prompts, plan)
            for name, tokens in prompts.items():
                zs.assert_logits_close(got[name], engine.plain(tokens), F32, name)
            engine.cache.check_consistency()
        assert engine.cache.stats().free_pages == (14, 8) and engine.cache.stats().free_slots == 2


def test_greedy_generation_through_the_scheduler():
    with ops.use(FakeOps()):
        parts = zs.ZuEngine(zs.MIXED, F32, "cpu", seed=31)
        engine = ContinuousBatchEngine.from_model(parts.model, block_size=8, total_blocks=96, max_running_requests=3,
                                                  max_batch_tokens=24, max_model_len=120)
        prompts = [zs.tokens_for(131, length, 40 + i) for i, length in enumerate([5, 37, 18, 2])]
        generated = engine.generate(prompts, max_new_tokens=6)
    for prompt, got in zip(prompts, generated):
        sequence = list(prompt)
        for _ in range(6):
            sequence.append(int(torch.argmax(parts.plain(sequence)[-1])))
        assert got == sequence[len(prompt):]


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed):
    config = zs.random_config(seed)
    with ops.use(FakeOps()):
        engine = zs.ZuEngine(config, F32, "cpu", seed=seed, num_pages=40)
        prompts = {"a": zs.tokens_for(config["vocab"], 45, seed), "b": zs.tokens_for(config["vocab"], 21, seed + 50)}
        got = engine.run_plan(prompts, [{"a": 17, "b": 1}, {"a": 1, "b": 2}, {"a": 2, "b": 18}, {"a": 25}])
    for name, tokens in prompts.items():
        zs.assert_logits_close(got[name], engine.plain(tokens), F32, f"seed {seed} {name}")
