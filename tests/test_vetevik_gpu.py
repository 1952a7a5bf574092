"""Vetevik through the framework's model, cache manager, step function and kernels, against the plain
implementation (``plain_vetevik``): each mechanism alone, whole prompts, token-by-token decoding, portions,
mixed batches, reused pages and slots, far keys, page borders and chunk edges with a key made to dominate, the
first tokens, long decoding through captured steps, odd and larger sizes, and greedy generation through the
scheduler and the command line."""

from __future__ import annotations

import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_vetevik as plain
import vetevik_support as vs
from mini_llm_runtime_b200 import ops
from mini_llm_runtime_b200.engine import ContinuousBatchEngine
from mini_llm_runtime_b200.ops.cuda_ops import AttentionBatch, plan_attention

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
F32 = torch.float32
F64 = torch.float64
BF16 = torch.bfloat16
DTYPES = [torch.float32, torch.bfloat16]


def run_alone(layer, dtype, seed=11, length=61, **options):
    config = vs.settled(vs.config([layer], width=72, vocab=90, **options), dtype)
    engine = vs.VEngine(config, dtype, DEVICE, seed=seed)
    tokens = vs.tokens_for(90, length, 5)
    want = engine.plain(tokens)
    vs.assert_logits_close(engine.run_cuts("a", tokens, []), want, dtype, "whole")
    vs.assert_logits_close(engine.run_cuts("b", tokens, [30] + list(range(31, length))), want, dtype, "decoded")
    vs.assert_logits_close(engine.run_cuts("c", tokens, [2, 17, 19, 40]), want, dtype, "portions")


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(6, 2, 16, 24), (3, 3, 10, 7), (1, 1, 8, 60), (8, 1, 12, 1), (4, 4, 40, 19), (4, 2, 32, 33), (2, 1, 64, 50)])
def test_attention_alone(sizes, dtype):
    run_alone(vs.attention(*sizes, scale=0.35, softcap=9.0), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 2, 16, 24, 3), (3, 3, 10, 7, 2), (1, 1, 8, 8, 1), (6, 1, 36, 20, 5), (2, 2, 64, 32, 4), (2, 1, 130, 12, 4)])
def test_delta_rule_alone(sizes, dtype):
    run_alone(vs.delta(*sizes), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("mlp", [vs.moe(56, 6, 1), vs.moe(56, 5, 3), vs.moe(64, 4, 2), vs.moe(24, 2, 2), vs.moe(20, 1, 1)])
def test_the_feed_forward(mlp, dtype):
    run_alone(vs.delta(2, 1, 8, 8, 2, mlp), dtype, seed=2, groups=2, mult=0.7)


@pytest.mark.parametrize("rows", [1, 7, 64, 65, 300])
@pytest.mark.parametrize("width,groups", [(72, 3), (64, 1), (70, 2), (4096, 4), (2560, 1)])
def test_the_stream_step_against_its_formula(rows, width, groups):
    """x += m * norm(delta), x += offset (a vector, rows, or none), norm of the new x, in parts of the row."""
    k = ops.current()
    generator = torch.Generator().manual_seed(rows + width)
    x, delta = torch.randn(rows, width, generator=generator), torch.randn(rows, width, generator=generator) * 3
    w1, w2 = 1 + 0.3 * torch.randn(width, generator=generator), 1 + 0.3 * torch.randn(width, generator=generator)
    for offset in (None, torch.randn(width, generator=generator), torch.randn(rows, width, generator=generator)):
        for with_delta in (True, False):
            want = x.double()
            if with_delta:
                want = want + plain.group_norm(delta.double(), w1.double(), 1e-5, groups)
            if offset is not None:
                want = want + offset.double()
            got_x = x.to(DEVICE)
            got = k.rms_norm_step(got_x, 1e-5, delta=delta.to(DEVICE) if with_delta else None, delta_weight=w1.to(DEVICE),
                                  norm_weight=w2.to(DEVICE), out_dtype=F32, groups=groups,
                                  offset=None if offset is None else offset.to(DEVICE))
            assert float((got_x.double().cpu() - want).abs().max()) < 2e-6 * float(want.abs().max())
            normed = plain.group_norm(want, w2.double(), 1e-5, groups)
            assert float((got.double().cpu() - normed).abs().max()) < 4e-6 * float(normed.abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("rows", [3, 40, 200])
@pytest.mark.parametrize("ff,width", [(64, 64), (128, 256), (72, 64), (20, 36)])
def test_experts_weighed_at_their_input(rows, ff, width, dtype):
    """Few rows (pairs one by one), many rows through the grouped product with and without the fused gate."""
    k = ops.current()
    generator = torch.Generator().manual_seed(rows + ff)
    experts, top = 5, 2
    x = torch.randn(rows, width, generator=generator).to(dtype)
    block = 64 if ff % 64 == 0 else ff
    gate = (torch.randn(experts, ff, width, generator=generator) * 2 / math.sqrt(width)).to(dtype)
    up = (torch.randn(experts, ff, width, generator=generator) / math.sqrt(width)).to(dtype)
    down = (torch.randn(experts, width, ff, generator=generator) / math.sqrt(ff)).to(dtype)
    stacked = torch.cat([gate.view(experts, -1, block, width), up.view(experts, -1, block, width)], dim=2).reshape(experts, 2 * ff, width)
    chosen = torch.stack([torch.randperm(experts, generator=generator)[:top] for _ in range(rows)]).to(torch.int32)
    weights = torch.rand(rows, top, generator=generator) * 2
    got = k.routed_experts(x.to(DEVICE), chosen.to(DEVICE), weights.to(DEVICE), stacked.contiguous().to(DEVICE), down.to(DEVICE),
                           block, "silu", weigh_input=True).double().cpu()
    want = torch.zeros(rows, width, dtype=F64)
    for r in range(rows):
        for t in range(top):
            e = int(chosen[r, t])
            h = weights[r, t].double() * x[r].double()
            want[r] += down[e].double() @ (plain.silu(gate[e].double() @ h) * (up[e].double() @ h))
    assert float((got - want).abs().max()) < (1e-5 if dtype == F32 else 2e-2) * float(want.abs().max())


def ragged_batch(lengths, starts, pages_per_request, generator):
    lengths, starts = np.array(lengths, dtype=np.int32), np.array(starts, dtype=np.int32)
    count = len(lengths)
    table = torch.randperm(count * pages_per_request, generator=generator).to(torch.int32).view(count, pages_per_request)
    row_start = np.concatenate([[0], np.cumsum(lengths)[:-1]]).astype(np.int32)
    arrays, counts = plan_attention(lengths, starts)

    def dev(a):
        return torch.as_tensor(a).to(device=DEVICE, dtype=torch.int32).contiguous()

    batch = AttentionBatch(dev(row_start), dev(lengths), dev(starts), dev(np.arange(count)), dev(table), count, int(lengths.max()),
                           int((starts + lengths).max()), {n: dev(v) for n, v in arrays.items()}, counts)
    return batch, lengths, starts, table, row_start


@pytest.mark.parametrize("page", [16, 24])
@pytest.mark.parametrize("heads,kv_heads,dim", [(4, 2, 64), (8, 1, 128), (40, 2, 32), (3, 3, 96), (6, 2, 40)])
@pytest.mark.parametrize("shape", [
    dict(chunk=130, softcap=5.0, slopes=True, sink=True, gate=True),       # scores several times the cap: tanh saturates
    dict(chunk=333, softcap=60.0, slopes=True, sink=True, gate=True),      # far below it: the series
    dict(chunk=0, softcap=0.0, slopes=False, sink=False, gate=False),      # ordinary softmax
    dict(chunk=0, softcap=8.0, slopes=True, sink=False, gate=True, window=77),
    dict(chunk=96, softcap=0.0, slopes=False, sink=True, gate=False, window=300),
])
def test_shaped_attention_kernels_against_their_formula(heads, kv_heads, dim, shape, page):
    """The float32 kernel, the bfloat16 kernel on the CUDA cores and (where the sizes allow it) the tensor-core
    kernels on a ragged batch over scattered pages: portions behind cached tokens and from the start, single
    rows, and a step of single rows only (which store their own keys)."""
    k = ops.current()
    generator = torch.Generator().manual_seed(heads * 100 + dim)
    chunk, window, softcap = shape["chunk"], shape.get("window", 0), shape["softcap"]
    scale = 3.0 / math.sqrt(dim)
    slopes = torch.rand(heads, generator=generator) * 0.2 if shape["slopes"] else None
    sink = torch.randn(heads, generator=generator) * 2 if shape["sink"] else None
    on_device = {"slopes": None if slopes is None else slopes.to(DEVICE), "sink": None if sink is None else sink.to(DEVICE)}
    group = heads // kv_heads
    for lengths, starts in (([70, 33, 1, 1, 2], [300, 0, 777, 64, 129]), ([1, 1, 1, 1], [0, 389, 390, 799])):
        batch, lengths, starts, table, row_start = ragged_batch(lengths, starts, -(-800 // page), generator)
        keys = torch.randn(len(lengths), 800, kv_heads, dim, generator=generator)
        rows = int(lengths.sum())
        width = (2 * heads + kv_heads) * dim
        projected = torch.randn(rows, width, generator=generator)
        for r in range(len(lengths)):      # the step's own keys
            projected[row_start[r]:row_start[r] + lengths[r], heads * dim:(heads + kv_heads) * dim] = \
                keys[r, starts[r]:starts[r] + lengths[r]].reshape(int(lengths[r]), -1)
        slots = torch.cat([table[r, (starts[r] + np.arange(lengths[r])) // page].long() * page + torch.from_numpy((starts[r] + np.arange(lengths[r])) % page)
                           for r in range(len(lengths))])
        for dtype, use_mma, limit in ((F32, False, 1e-5), (BF16, False, 1e-2), (BF16, True, 1e-2)):
            pool = torch.zeros(table.numel(), kv_heads, page, dim, dtype=dtype)
            for r in range(len(lengths)):
                before = torch.arange(int(starts[r]))      # what earlier steps left; the step's own keys are not there yet
                pool[table[r, before // page].long(), :, before % page] = keys[r, :int(starts[r])].to(dtype)
            pool = pool.to(DEVICE)
            x = projected.to(dtype)
            xd = x.to(DEVICE)
            gate = xd[:, (heads + kv_heads) * dim:] if shape["gate"] else None
            k.use_mma_attention = use_mma
            try:
                got = k.shaped_attention(xd[:, :heads * dim], xd[:, heads * dim:(heads + kv_heads) * dim], None, slots.to(DEVICE), pool,
                                         None, batch, heads, kv_heads, dim, dim, scale, softcap=softcap, window=window, chunk=chunk,
                                         gate=gate, **on_device)
            finally:
                k.use_mma_attention = True
            got, stored = got.double().cpu(), pool.cpu()
            for r in range(len(lengths)):
                for i in range(int(lengths[r])):
                    position, row = int(starts[r]) + i, int(row_start[r]) + i
                    assert torch.equal(stored[int(slots[row]) // page, :, int(slots[row]) % page], keys[r, position].to(dtype))
                    lo = max(position // chunk * chunk if chunk else 0, position - window + 1 if window else 0)
                    kk = keys[r, lo:position + 1].to(dtype).double().repeat_interleave(group, dim=1)
                    score = torch.einsum("hd,khd->hk", x[row, :heads * dim].double().view(heads, dim), kk) * scale
                    if softcap:
                        score = softcap * torch.tanh(score / softcap)
                    if slopes is not None:
                        score = score - slopes.double()[:, None] * (position - torch.arange(lo, position + 1)).double()[None]
                    if sink is not None:
                        score = torch.cat([score, sink.double()[:, None]], dim=1)
                    p = torch.softmax(score, dim=-1)[:, :position + 1 - lo]
                    want = torch.einsum("hk,khd->hd", p, kk).reshape(-1)
                    if shape["gate"]:
                        want = want * torch.sigmoid(x[row, (heads + kv_heads) * dim:].double())
                    error = float((got[row] - want).abs().max()) / max(float(want.abs().max()), 0.1)
                    assert error < limit, f"{dtype}, tensor cores {use_mma}: request {r}, row {i}: off by {error:.2e}"


def test_shaped_attention_with_values_of_their_own():
    """Keys and values apart, of different sizes, through the part's own kernels (no layer of Vetevik asks for
    it)."""
    k = ops.current()
    generator = torch.Generator().manual_seed(8)
    heads, kv_heads, dim, vdim, page = 4, 2, 24, 40, 16
    batch, lengths, starts, table, row_start = ragged_batch([20, 1], [0, 0], 4, generator)
    x = torch.randn(21, heads * dim + kv_heads * (dim + vdim), generator=generator)
    slots = torch.cat([table[r, np.arange(lengths[r]) // page].long() * page + torch.from_numpy(np.arange(lengths[r]) % page)
                       for r in range(2)])
    k_pool = torch.zeros(table.numel(), kv_heads, page, dim, device=DEVICE)
    v_pool = torch.zeros(table.numel(), kv_heads, page, vdim, device=DEVICE)
    xd = x.to(DEVICE)
    a, b = heads * dim, (heads + kv_heads) * dim
    got = k.shaped_attention(xd[:, :a], xd[:, a:b], xd[:, b:], slots.to(DEVICE), k_pool, v_pool, batch, heads, kv_heads, dim, vdim,
                             0.3, softcap=5.0, chunk=7).double().cpu()
    for i in range(20):
        lo = i // 7 * 7
        kk = x[lo:i + 1, a:b].double().view(-1, kv_heads, dim).repeat_interleave(2, dim=1)
        vv = x[lo:i + 1, b:].double().view(-1, kv_heads, vdim).repeat_interleave(2, dim=1)
        score = 5.0 * torch.tanh(torch.einsum("hd,khd->hk", x[i, :a].double().view(heads, dim), kk) * 0.3 / 5.0)
        want = torch.einsum("hk,khd->hd", torch.softmax(score, dim=-1), vv).reshape(-1)
        assert float((got[i] - want).abs().max()) < 1e-5


@pytest.mark.parametrize("heads,kv_heads,dim,vdim,taps", [(4, 2, 32, 24, 3), (3, 3, 64, 40, 4), (4, 1, 128, 36, 2), (2, 1, 200, 16, 4),
                                                          (2, 2, 384, 12, 4), (2, 1, 10, 6, 1), (3, 1, 66, 33, 5), (2, 2, 256, 20, 2)])
def test_delta_kernels_against_their_formulas(heads, kv_heads, dim, vdim, taps):
    """Convolution, recurrence and gated head norm on a ragged batch whose requests go on over several steps with
    portions of every remainder of the kernel's block of tokens; decays from about 0 to about 1."""
    k = ops.current()
    generator = torch.Generator().manual_seed(dim + vdim)
    qk, inner = kv_heads * dim, heads * vdim
    channels = 2 * qk + inner
    width = channels + inner + 2 * heads + (-(channels + inner + 2 * heads)) % 8
    conv = torch.randn(channels, taps, generator=generator) * 0.7
    dt_bias, a_log = torch.randn(heads, generator=generator), torch.linspace(-6.0, 3.0, heads)
    weight = 1 + 0.2 * torch.randn(vdim, generator=generator)
    lengths = [[37, 1, 2, 64], [1, 3, 41, 5], [1, 1, 1, 1], [6, 70, 4, 1]]
    total = [sum(col) for col in zip(*lengths)]
    sequences = [torch.randn(t, width, generator=generator) for t in total]
    conv_state = torch.zeros(4, taps - 1, channels, device=DEVICE)
    state = torch.zeros(4, heads, vdim, dim, device=DEVICE)
    done, got = [0] * 4, [[] for _ in range(4)]
    at = channels + inner
    for step in lengths:
        rows = torch.cat([sequences[i][done[i]:done[i] + step[i]] for i in range(4)]).to(DEVICE)
        first = np.concatenate([[0], np.cumsum(step)[:-1]])
        ctx = SimpleNamespace(seg_q_start=torch.tensor(first, dtype=torch.int32, device=DEVICE),
                              seg_q_len=torch.tensor(step, dtype=torch.int32, device=DEVICE),
                              seg_slot=torch.tensor([2, 0, 3, 1], dtype=torch.int32, device=DEVICE), num_segments=4, max_q_len=max(step))
        mixed = k.causal_conv(rows[:, :channels], conv.to(DEVICE), None, conv_state, ctx, "silu")
        y = k.delta_rule_scan(mixed[:, :qk], mixed[:, qk:2 * qk], mixed[:, 2 * qk:], rows[:, at:at + heads],
                              rows[:, at + heads:at + 2 * heads], dt_bias.to(DEVICE), a_log.to(DEVICE), state, ctx, heads, kv_heads, dim,
                              vdim, 1e-6)
        out = k.gated_head_norm(y, rows[:, channels:at], weight.to(DEVICE), 1e-5, heads, F32)
        for i in range(4):
            got[i].append(out[first[i]:first[i] + step[i]].cpu())
            done[i] += step[i]
    for i in range(4):
        u = sequences[i].double()
        mixed = plain.short_conv(u[:, :channels], conv.double())
        q = plain.unit(mixed[:, :qk].view(-1, kv_heads, dim)) * dim ** -0.5
        kk = plain.unit(mixed[:, qk:2 * qk].view(-1, kv_heads, dim))
        v = mixed[:, 2 * qk:].view(-1, heads, vdim)
        decay = torch.exp(-torch.exp(a_log.double()) * torch.nn.functional.softplus(u[:, at:at + heads] + dt_bias.double()))
        beta = torch.sigmoid(u[:, at + heads:at + 2 * heads])
        want = torch.zeros(total[i], heads, vdim, dtype=F64)
        for h in range(heads):
            kv = h // (heads // kv_heads)
            want[:, h] = plain.delta_recurrence(q[:, kv], kk[:, kv], v[:, h], decay[:, h], beta[:, h])
        want = (plain.rms(want, 1e-5) * weight.double() * plain.silu(u[:, channels:at]).view(-1, heads, vdim)).reshape(total[i], inner)
        error = float((torch.cat(got[i]).double() - want).abs().max()) / float(want.abs().max())
        assert error < 3e-5, f"request {i}: off by {error:.2e}"


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["MIXED", "ODD", "PLAIN"])
def test_prefill_against_token_by_token(name, dtype):
    config = vs.settled(getattr(vs, name), dtype)
    engine = vs.VEngine(config, dtype, DEVICE, seed=({"MIXED": 14, "ODD": 16, "PLAIN": 1} if dtype == F32 else {"MIXED": 12, "ODD": 8, "PLAIN": 1})[name])
    tokens = vs.tokens_for(config["vocab"], 75, 8)
    want = engine.plain(tokens)
    # heads of five to ten entries: a rounding weighs more
    spread = 8e-2 if name == "ODD" else 4e-2
    for what, cuts in (("whole", []), ("token by token", range(1, 75)), ("prompt then decode", [40] + list(range(41, 75)))):
        vs.assert_logits_close(engine.run_cuts(what, tokens, cuts), want, dtype, what, spread)


@pytest.mark.parametrize("cuts", [[2, 4, 6, 8], [3, 19, 20, 52], [16, 32, 48, 64], [1, 2, 35, 37, 90], [21, 42, 50, 63]])
def test_portions_of_several_sizes(cuts):
    engine = vs.VEngine(vs.MIXED, F32, DEVICE, seed=1)
    tokens = vs.tokens_for(131, 100, 9)
    vs.assert_logits_close(engine.run_cuts("a", tokens, cuts), engine.plain(tokens), F32)


def test_float32_logits_do_not_depend_on_the_cut():
    engine = vs.VEngine(vs.MIXED, F32, DEVICE, seed=1)
    tokens = vs.tokens_for(131, 90, 10)
    whole = engine.run_cuts("a", tokens, [])
    pieces = engine.run_cuts("b", tokens, [2, 5, 30, 31, 64])
    assert float((whole - pieces).abs().max()) <= 2e-5 * float(whole.abs().max())


def test_the_first_tokens_of_a_sequence():
    engine = vs.VEngine(vs.MIXED, F32, DEVICE, seed=14)
    for length in (1, 2, 3, 13):
        tokens = vs.tokens_for(131, length, length)
        want = engine.plain(tokens)
        vs.assert_logits_close(engine.run_cuts("p", tokens, []), want, F32, f"prompt of {length}")
        vs.assert_logits_close(engine.run_cuts("d", tokens, range(1, length)), want, F32, f"decoded from the first token, {length}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests(dtype):
    engine = vs.VEngine(vs.settled(vs.MIXED, dtype), dtype, DEVICE, seed=7, num_pages=40)
    prompts = {"a": vs.tokens_for(131, 70, 1), "b": vs.tokens_for(131, 41, 2), "c": vs.tokens_for(131, 9, 3),
               "d": vs.tokens_for(131, 100, 4)}
    plan = [{"a": 30, "b": 1, "d": 2}, {"a": 1, "b": 16, "c": 9, "d": 50}, {"a": 1, "b": 1, "d": 1},
            {"a": 38, "b": 23, "d": 47}]
    got = engine.run_plan(prompts, plan)
    for name, tokens in prompts.items():
        vs.assert_logits_close(got[name], engine.plain(tokens), dtype, name)


def test_pages_and_slots_are_used_again():
    """Two slots and few pages serve six requests in turn: a slot's states start at zero again, pages of chunks
    that have passed are taken by others, and pages written by one request are read by the next."""
    config = vs.config([vs.delta(2, 1, 8, 12, 3, vs.moe(24, 4, 2)), vs.attention(4, 2, 6, 11), vs.attention(2, 2, 10, 30)],
                       width=40, vocab=70, groups=2, mult=0.8, loop=(0, 2, 2))
    slow = {"l0.mix.A_log": lambda t: torch.full_like(t, -7.0)}       # a state left behind would stay for long
    engine = vs.VEngine(config, F32, DEVICE, seed=16, page_size=8, num_pages=[8, 14], max_requests=2, max_tokens=64,
                        max_step_tokens=16, overrides=slow)
    for number in range(3):
        prompts = {f"a{number}": vs.tokens_for(70, 33 + 7 * number, 20 + number), f"b{number}": vs.tokens_for(70, 25, 30 + number)}
        plan = []
        for start in range(0, 60, 6):
            step = {name: min(6, len(tokens) - start) for name, tokens in prompts.items() if start < len(tokens)}
            if step:
                plan.append(step)
        got = engine.run_plan(prompts, plan)
        for name, tokens in prompts.items():
            vs.assert_logits_close(got[name], engine.plain(tokens), F32, name)
        engine.cache.check_consistency()
    assert engine.cache.stats().free_pages == (8, 14)


@pytest.mark.parametrize("dtype,dim,kv_heads", [(F32, 48, 1), (BF16, 64, 2)])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portions"])
@pytest.mark.parametrize("query,key,chunk", [
    (290, 2, 1000),      # a key far back among hundreds
    (271, 15, 300),      # far back, at the last place of a page
    (64, 63, 300),       # the neighbour, across a page's and a tile's border
    (48, 32, 300),       # a page's first place
    (5, 0, 300),         # the very first token
    (299, 150, 150),     # the first key of the query's chunk, seen by the chunk's last position
    (299, 149, 150),     # the last key of the chunk before: not seen
    (150, 149, 150),     # the chunk's first position does not see its neighbour
    (150, 150, 150),     # it sees itself only
    (257, 192, 64),      # one chunk too far, chunks that end with tiles
    (255, 192, 64),      # just inside
    (131, 125, 7),       # chunks shorter than a page
    (131, 126, 7),
])
def test_far_keys_page_borders_and_chunk_edges_with_a_dominant_key(query, key, chunk, how, dtype, dim, kv_heads):
    length = 300
    config, overrides = vs.dominant_key_case(length, query, key, chunk, seed=query + key, dim=dim, kv_heads=kv_heads)
    engine = vs.VEngine(config, dtype, DEVICE, seed=5, overrides=overrides, num_pages=24, max_tokens=320)
    tokens = list(range(length))
    want = engine.plain(tokens)
    cuts = {"prompt": [], "decoded": [3] + list(range(4, length)), "portions": [2, max(3, query - 1), query, min(query + 2, length)]}[how]
    got = engine.run_cuts("a", tokens, cuts)
    vs.assert_logits_close(got[query:query + 1], want[query:query + 1], dtype, f"query {query}")
    vs.assert_logits_close(got, want, dtype)
    if key == query:
        return
    # the case tells: with another token at the key's place, the answer at the query differs exactly if it is seen
    hidden = list(tokens)
    hidden[key] = (key + 101) % length
    change = float((engine.plain(hidden)[query] - want[query]).abs().max()) / float(want[query].abs().max())
    if query // chunk == key // chunk:
        assert change > 0.1
    else:
        assert change < 1e-12
        # and a chunk that reached that far would show
        wider = json.loads(json.dumps(config))
        wider["layers"][0]["mixer"]["mask"]["size"] = 1000
        seen = engine.plain(tokens, config_dict=wider)
        assert float((seen[query] - want[query]).abs().max()) > 0.1 * float(want[query].abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_captured_steps(dtype):
    engine = vs.VEngine(vs.settled(vs.MIXED, dtype), dtype, DEVICE, seed=14 if dtype == F32 else 12, num_pages=64)
    tokens = vs.tokens_for(131, 260, 13)
    want = engine.plain(tokens)
    got = engine.run_cuts("a", tokens, [30] + list(range(31, 260)))
    assert engine.runner.graph_replays > 100
    vs.assert_logits_close(got, want, dtype)
    other = vs.tokens_for(131, 60, 14)
    engine.cache.create_request("x")
    engine.cache.create_request("y")
    first = engine.step([("x", tokens[:20], range(20)), ("y", other[:10], range(10))])
    rows = {"x": [first[:20]], "y": [first[20:]]}
    for i in range(40):
        logits = engine.step([("x", tokens[20 + i:21 + i], [0]), ("y", other[10 + i:11 + i], [0])])
        rows["x"].append(logits[:1])
        rows["y"].append(logits[1:])
    vs.assert_logits_close(torch.cat(rows["x"]), vs.take(want, slice(0, 60)), dtype, "x")
    vs.assert_logits_close(torch.cat(rows["y"]), engine.plain(other[:50]), dtype, "y")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_the_tensor_core_kernels_take(dtype):
    engine = vs.VEngine(vs.settled(vs.WIDE, dtype), dtype, DEVICE, seed=14, num_pages=80, max_tokens=1024)
    tokens = vs.tokens_for(520, 420, 22)
    want = engine.plain(tokens)
    vs.assert_logits_close(engine.run_cuts("a", tokens, [300, 301, 302, 350]), want, dtype)
    prompts = {"p": tokens[:200], "q": vs.tokens_for(520, 150, 24)}
    got = engine.run_plan(prompts, [{"p": 130, "q": 1}, {"p": 1, "q": 140}, {"p": 69, "q": 9}])
    vs.assert_logits_close(got["p"], vs.take(want, slice(0, 200)), dtype, "p")
    vs.assert_logits_close(got["q"], engine.plain(prompts["q"]), dtype, "q")


@pytest.mark.parametrize("seed", range(6))
def test_configurations_drawn_at_random(seed):
    config = vs.random_config(seed + 100)
    engine = vs.VEngine(config, F32, DEVICE, seed=seed, num_pages=40)
    prompts = {"a": vs.tokens_for(config["vocab"], 45, seed), "b": vs.tokens_for(config["vocab"], 21, seed + 50)}
    got = engine.run_plan(prompts, [{"a": 17, "b": 1}, {"a": 1, "b": 2}, {"a": 2, "b": 18}, {"a": 25}])
    for name, tokens in prompts.items():
        vs.assert_logits_close(got[name], engine.plain(tokens), F32, f"seed {seed} {name}")


def test_greedy_generation_through_the_scheduler():
    parts = vs.VEngine(vs.MIXED, F32, DEVICE, seed=31)
    engine = ContinuousBatchEngine.from_model(parts.model, block_size=8, total_blocks=96, max_running_requests=3,
                                              max_batch_tokens=24, max_model_len=160)
    prompts = [vs.tokens_for(131, length, 40 + i) for i, length in enumerate([5, 37, 18, 50, 2])]
    generated = engine.generate(prompts, max_new_tokens=12)
    for prompt, got in zip(prompts, generated):
        sequence = list(prompt)
        for _ in range(12):
            sequence.append(int(torch.argmax(parts.plain(sequence)[-1])))
        assert got == sequence[len(prompt):]


def test_command_line_and_replay_program_with_a_model_folder(tmp_path):
    """``make-random`` writes a Vetevik folder from a config.json, ``generate`` reproduces the plain
    implementation's greedy tokens from it, and the replay program writes the logits of the wanted places step
    by step, with pages and slots given back in between."""
    import os
    import subprocess
    import sys

    from mini_llm_runtime_b200.weights import read_checkpoint

    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    env = dict(os.environ, PYTHONPATH=root + os.pathsep + os.environ.get("PYTHONPATH", ""))

    def cli(*arguments, stdin=None):
        done = subprocess.run([sys.executable, *arguments], capture_output=True, text=True, env=env, timeout=600,
                              input=stdin)
        assert done.returncode == 0, done.stderr[-2000:]
        return done.stdout

    (tmp_path / "config.json").write_text(json.dumps(vs.MIXED))
    folder = tmp_path / "model"
    cli("-m", "mini_llm_runtime_b200", "make-random", "--config", str(tmp_path / "config.json"), "--seed", "4",
        "--out", str(folder))
    tensors = read_checkpoint(folder)
    prompt = vs.tokens_for(131, 11, 6)
    sequence = list(prompt)
    for _ in range(5):
        sequence.append(int(torch.argmax(plain.forward(vs.MIXED, tensors, sequence)[0][-1])))
    record = json.loads(cli("-m", "mini_llm_runtime_b200", "generate", "--model", str(folder), "--dtype", "float32",
                            "--max-model-len", "64", "--prompt-ids", ",".join(map(str, prompt)), "--max-new-tokens", "5"
                            ).splitlines()[-1])
    assert record["generated_ids"] == sequence[len(prompt):]

    other = vs.tokens_for(131, 30, 7)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": prompt[:4], "want": [0, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": prompt[4:], "want": [6]},
                                     {"id": "o", "tokens": other, "want": [29]}], "end": ["p"]},
             {"step": 2, "entries": [], "end": ["o"]}]
    out = cli(os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out",
              str(tmp_path / "logits"), "--max-tokens", "64", stdin="\n".join(json.dumps(s) for s in steps) + "\n")
    assert [line for line in out.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    first = torch.from_numpy(np.fromfile(tmp_path / "logits" / "0.f32", dtype="<f4").reshape(2, 131))
    second = torch.from_numpy(np.fromfile(tmp_path / "logits" / "1.f32", dtype="<f4").reshape(2, 131))
    want = plain.forward(vs.MIXED, tensors, prompt)[0]
    vs.assert_logits_close(torch.cat([first, second[:1]]), want[[0, 3, 10]], F32)
    vs.assert_logits_close(second[1:], plain.forward(vs.MIXED, tensors, other)[0][29:], F32)
