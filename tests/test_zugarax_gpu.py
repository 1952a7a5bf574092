"""Zugarax through the framework's model, cache manager, step function and kernels, against the plain implementation
(``plain_zugarax``): each mechanism alone, kernels against their formulas, whole prompts, token-by-token decoding,
portions, mixed batches, reused pages and slots, far keys, page borders and window edges with a key made to dominate,
the first tokens, long decoding through captured steps, odd and larger sizes, and greedy generation through the
scheduler and the command line."""

from __future__ import annotations

import json
import math
from types import SimpleNamespace

import numpy as np
import pytest
import torch

import plain_zugarax as plain
import zugarax_support as zs
from mini_llm_runtime_b200 import ops
from mini_llm_runtime_b200.engine import ContinuousBatchEngine
from mini_llm_runtime_b200.ops.cuda_ops import AttentionBatch, plan_attention

pytestmark = pytest.mark.gpu

DEVICE = "cuda:0"
F32 = torch.float32
F64 = torch.float64
BF16 = torch.bfloat16
DTYPES = [torch.float32, torch.bfloat16]


def run_alone(layers, dtype, seed=11, length=61, **options):
    layers = layers if isinstance(layers, list) else [layers]
    engine = zs.ZuEngine(zs.config(layers, width=72, vocab=90, **options), dtype, DEVICE, seed=seed)
    tokens = zs.tokens_for(90, length, 5)
    want = engine.plain(tokens)
    zs.assert_logits_close(engine.run_cuts("a", tokens, []), want, dtype, "whole")
    zs.assert_logits_close(engine.run_cuts("b", tokens, [30] + list(range(31, length))), want, dtype, "decoded")
    zs.assert_logits_close(engine.run_cuts("c", tokens, [2, 17, 19, 40]), want, dtype, "portions")


# ---------------------------------------------------------------- each mechanism alone
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes,rot", [
    ((6, 2, 16, 16, 24), zs.rotation(50.0, 8, zs.bands(4.0, 1.0, 3.0, 40))), ((3, 3, 10, 14, 7), zs.rotation(9.0, 2)),
    ((1, 1, 8, 8, 60), zs.rotation(100.0, 8)), ((8, 1, 12, 20, 1), zs.rotation(20.0, 6)), ((4, 4, 40, 40, 19), zs.rotation(1e4, 40)),
    ((4, 2, 32, 32, 33), zs.rotation(300.0, 16, zs.bands(2.0, 1.0, 9.0, 70))), ((2, 1, 64, 64, 2), zs.rotation(1e3, 64)),
    ((2, 1, 64, 32, 50), zs.rotation(1e3, 24))])
def test_windowed_attention_alone(sizes, rot, dtype):
    run_alone(zs.attention(*sizes, rot, scale=0.35), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 16, 8, 16, 24), (3, 10, 6, 7, 20), (1, 8, 2, 8, 8), (6, 12, 16, 20, 64), (2, 64, 32, 64, 128), (18, 8, 8, 8, 32)])
def test_latent_attention_alone_and_shared(sizes, dtype):
    options = dict(base=300.0, scaling=zs.ramp(3.0, 50, 8.0, 1.0))
    heads, dim, rot_dim, vdim, rank = sizes
    run_alone(zs.latent(*sizes, **options), dtype)
    run_alone([zs.latent(*sizes, **options), zs.latent(heads + 1, dim + 8, rot_dim, vdim + 4, rank, **options, kv_from=0)], dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("sizes", [(4, 16, 24), (3, 10, 7), (1, 8, 8), (6, 36, 20), (2, 64, 32), (2, 130, 12), (2, 128, 128), (1, 6, 1)])
@pytest.mark.parametrize("cap", [3.0, 18.0])
def test_matrix_memory_alone(sizes, cap, dtype):
    run_alone(zs.mlstm(*sizes, cap), dtype)


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("ff,limit", [(56, 0.7), (64, 1.0), (128, 3.0), (20, 0.3)])
def test_the_feed_forward_with_biases(ff, limit, dtype):
    run_alone(zs.mlstm(2, 8, 8, 5.0, zs.dense(ff, limit)), dtype, seed=2, scale=2.0)


# ---------------------------------------------------------------- kernels against their formulas
@pytest.mark.parametrize("rows", [3, 40, 100, 200, 500])
@pytest.mark.parametrize("ff,width", [(64, 64), (384, 256), (72, 64), (2048, 512)])
def test_clamped_gate_with_biases(rows, ff, width):
    """Few rows (a kernel of its own behind the product), and every epilogue of the tensor-core product."""
    k = ops.current()
    generator = torch.Generator().manual_seed(rows + ff)
    block = 64 if ff % 64 == 0 else ff
    for dtype in DTYPES:
        x = torch.randn(rows, width, generator=generator).to(dtype)
        gate, up = ((torch.randn(ff, width, generator=generator) / math.sqrt(width)).to(dtype) for _ in range(2))
        gate_b, up_b = (torch.randn(ff, generator=generator).to(dtype) for _ in range(2))
        weight = torch.cat([gate.view(-1, block, width), up.view(-1, block, width)], dim=1).reshape(2 * ff, width).contiguous()
        bias = torch.cat([gate_b.view(-1, block), up_b.view(-1, block)], dim=1).reshape(-1)
        got = k.linear_clamped_gate(x.to(DEVICE), weight.to(DEVICE), block, 1.1, 1.702, bias=bias.to(DEVICE)).double().cpu()
        g = (x.double() @ gate.double().T + gate_b.double()).clamp(max=1.1)
        u = (x.double() @ up.double().T + up_b.double()).clamp(-1.1, 1.1)
        want = g * torch.sigmoid(1.702 * g) * (u + 1.0)
        assert float((got - want).abs().max()) < (1e-5 if dtype == F32 else 2e-2) * float(want.abs().max())


@pytest.mark.parametrize("count", [5, 1000, 70001])
def test_capped_logits(count):
    x = torch.randn(count, generator=torch.Generator().manual_seed(count)) * 20
    got = ops.current().softcap_(x.to(DEVICE), 7.5).double().cpu()
    assert float((got - 7.5 * torch.tanh(x.double() / 7.5)).abs().max()) < 2e-6


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("heads,kv_heads,dim,vdim,rot", [(4, 2, 64, 64, 32), (3, 1, 128, 96, 128), (5, 5, 10, 7, 6), (2, 2, 200, 40, 8),
                                                         (8, 2, 32, 32, 4), (2, 1, 16, 12, 0), (1, 1, 4, 4, 2)])
@pytest.mark.parametrize("interleaved", [False, True])
def test_head_prepare_against_its_formula(heads, kv_heads, dim, vdim, rot, interleaved, dtype):
    k = ops.current()
    generator = torch.Generator().manual_seed(dim + heads)
    rows, page = 23, 8
    width = (heads + kv_heads) * dim + kv_heads * vdim + 8
    x = torch.randn(rows, width, generator=generator).to(dtype)
    positions = torch.randint(0, 5000, (rows,), generator=generator).to(torch.int32)
    slots = torch.randperm(64, generator=generator)[:rows]
    slots[3] = -1                                   # a row whose key and value are not stored
    freq = torch.rand(rot // 2, generator=generator) if rot else None
    wq, wk = (1 + 0.3 * torch.randn(dim, generator=generator) for _ in range(2))
    a, b = heads * dim, (heads + kv_heads) * dim
    xd = x.to(DEVICE)
    for with_norm in (True, False):
        k_pool = torch.zeros(8, kv_heads, page, dim, dtype=dtype, device=DEVICE)
        v_pool = torch.zeros(8, kv_heads, page, vdim, dtype=dtype, device=DEVICE)
        q = k.head_prepare(xd[:, :a], xd[:, a:b], xd[:, b:b + kv_heads * vdim], positions.to(DEVICE),
                           wq.to(DEVICE) if with_norm else None, wk.to(DEVICE) if with_norm else None, 1e-5,
                           None if freq is None else freq.to(DEVICE), 1.3, interleaved, slots.to(DEVICE), k_pool, v_pool,
                           heads, kv_heads, dim, vdim).cpu()

        def prepared(part, count, weight):
            y = part.double().view(rows, count, dim)
            if with_norm:
                y = plain.rms(y, 1e-5) * weight.double()
            if rot:
                angle = (positions.float()[:, None] * freq[None, :]).double()      # angles are 32-bit
                cos, sin = torch.cos(angle)[:, None] * 1.3, torch.sin(angle)[:, None] * 1.3
                first = torch.arange(rot // 2) * (2 if interleaved else 1)
                second = first + (1 if interleaved else rot // 2)
                z = y.clone()
                z[..., first] = y[..., first] * cos - y[..., second] * sin
                z[..., second] = y[..., second] * cos + y[..., first] * sin
                y = z
            return y

        limit = 3e-6 if dtype == F32 else 8e-3
        want_q, want_k = prepared(x[:, :a], heads, wq), prepared(x[:, a:b], kv_heads, wk)
        assert float((q.double().view(rows, heads, dim) - want_q).abs().max()) < limit * float(want_q.abs().max())
        keys, values = k_pool.cpu(), v_pool.cpu()
        for r in range(rows):
            if int(slots[r]) < 0:
                continue
            at, offset = divmod(int(slots[r]), page)
            assert float((keys[at, :, offset].double() - want_k[r]).abs().max()) < limit * float(want_k.abs().max())
            assert torch.equal(values[at, :, offset], x[r, b:b + kv_heads * vdim].view(kv_heads, vdim))
        assert int((keys.abs().sum(dim=(1, 3)) > 0).sum()) == rows - 1


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
@pytest.mark.parametrize("heads,kv_heads,dim,vdim", [(4, 2, 64, 64), (8, 1, 128, 128), (40, 2, 32, 32), (3, 3, 96, 96), (6, 2, 40, 24)])
@pytest.mark.parametrize("window", [1, 77, 300, 0])
def test_windowed_attention_over_values_of_their_own(heads, kv_heads, dim, vdim, window, page):
    """Keys and values already in scattered pages, a sink of score zero, an output gate: portions behind cached tokens
    and from the start, single rows, and a step of single rows only, through the float32 kernel, the bfloat16 kernel
    on the CUDA cores and (where the sizes allow it) the tensor-core kernels."""
    k = ops.current()
    generator = torch.Generator().manual_seed(heads * 100 + dim)
    scale, group = 2.0 / math.sqrt(dim), heads // kv_heads
    sink = torch.zeros(heads, device=DEVICE)
    for lengths, starts in (([70, 33, 1, 1, 2], [300, 0, 777, 64, 129]), ([1, 1, 1, 1], [0, 389, 390, 799])):
        batch, lengths, starts, table, row_start = ragged_batch(lengths, starts, -(-800 // page), generator)
        keys, values = (torch.randn(len(lengths), 800, kv_heads, n, generator=generator) for n in (dim, vdim))
        rows = int(lengths.sum())
        q32 = torch.randn(rows, heads * dim, generator=generator)
        gate32 = torch.randn(rows, heads * vdim + 4, generator=generator)      # a view with a stride of its own
        for dtype, use_mma, limit in ((F32, False, 1e-5), (BF16, False, 1e-2), (BF16, True, 1e-2)):
            k_pool = torch.full((table.numel(), kv_heads, page, dim), 100.0, dtype=dtype)      # keys nobody may see
            v_pool = torch.full((table.numel(), kv_heads, page, vdim), 100.0, dtype=dtype)
            for r in range(len(lengths)):
                seen = torch.arange(int(starts[r] + lengths[r]))
                at, offset = table[r, seen // page].long(), seen % page
                k_pool[at, :, offset] = keys[r, seen].to(dtype)
                v_pool[at, :, offset] = values[r, seen].to(dtype)
            q, gate = q32.to(dtype), gate32.to(dtype)
            k.use_mma_attention = use_mma
            try:
                got = k.shaped_attention(q.to(DEVICE), None, None, torch.zeros(rows, dtype=torch.int64, device=DEVICE), k_pool.to(DEVICE),
                                         v_pool.to(DEVICE), batch, heads, kv_heads, dim, vdim, scale, window=window, sink=sink,
                                         gate=gate.to(DEVICE)[:, :heads * vdim], write_kv=False)
            finally:
                k.use_mma_attention = True
            got = got.double().cpu()
            for r in range(len(lengths)):
                for i in range(int(lengths[r])):
                    position, row = int(starts[r]) + i, int(row_start[r]) + i
                    lo = max(0, position - window + 1) if window else 0
                    kk = keys[r, lo:position + 1].to(dtype).double().repeat_interleave(group, dim=1)
                    vv = values[r, lo:position + 1].to(dtype).double().repeat_interleave(group, dim=1)
                    e = torch.exp(torch.einsum("hd,khd->hk", q[row].double().view(heads, dim), kk) * scale)
                    want = torch.einsum("hk,khd->hd", e / (1.0 + e.sum(dim=1, keepdim=True)), vv).reshape(-1)
                    want = want * torch.sigmoid(gate[row, :heads * vdim].double())
                    error = float((got[row] - want).abs().max()) / max(float(want.abs().max()), 0.1)
                    assert error < limit, f"{dtype}, tensor cores {use_mma}: request {r}, row {i}: off by {error:.2e}"


@pytest.mark.parametrize("heads,dim,vdim", [(4, 32, 24), (3, 64, 40), (4, 128, 36), (2, 200, 16), (2, 384, 12), (2, 10, 6), (3, 66, 33),
                                            (2, 256, 20), (2, 128, 128), (1, 40, 300), (3, 64, 64), (2, 128, 24), (5, 64, 40)])
@pytest.mark.parametrize("dtype", DTYPES)
def test_matrix_memory_kernels_against_their_formula(heads, dim, vdim, dtype):
    """A ragged batch whose requests go on over several steps with portions of every remainder of the kernels' blocks
    and chunks of tokens, and steps of single rows; gates from shut to wide open, over long and short memories; in
    bfloat16 the sizes of 64 and 128 go through the tensor cores."""
    k = ops.current()
    generator = torch.Generator().manual_seed(dim + vdim)
    qk, inner, cap = heads * dim, heads * vdim, 9.0
    width = 2 * qk + 2 * inner + 2 * heads
    width += -width % 8
    lengths = [[37, 1, 2, 300], [1, 3, 41, 5], [1, 1, 1, 1], [6, 70, 4, 1], [1, 1, 1, 1], [64, 128, 65, 63]]
    total = [sum(col) for col in zip(*lengths)]
    sequences = [torch.randn(t, width, generator=generator) for t in total]
    at = 2 * qk + 2 * inner
    for i, sequence in enumerate(sequences):
        sequence[:, at:at + heads] *= (1.0, 8.0, 3.0, 5.0)[i]
        sequence[:, at + heads:at + 2 * heads] = sequence[:, at + heads:at + 2 * heads] * 2.0 + (6.0, 0.0, -3.0, 4.0)[i]
        if dtype == BF16:      # projections may be rounded on their way into the products
            sequence[:, :2 * qk + inner] = sequence[:, :2 * qk + inner].to(BF16).float()
    i_bias, f_bias = torch.randn(heads, generator=generator), torch.randn(heads, generator=generator)
    weight = 1 + 0.2 * torch.randn(inner, generator=generator)
    state, maximum = torch.zeros(4, heads, vdim + 1, dim, device=DEVICE), torch.zeros(4, heads, device=DEVICE)
    done, got = [0] * 4, [[] for _ in range(4)]
    for step in lengths:
        rows = torch.cat([sequences[i][done[i]:done[i] + step[i]] for i in range(4)]).to(DEVICE)
        first = np.concatenate([[0], np.cumsum(step)[:-1]])
        ctx = SimpleNamespace(seg_q_start=torch.tensor(first, dtype=torch.int32, device=DEVICE),
                              seg_q_len=torch.tensor(step, dtype=torch.int32, device=DEVICE),
                              seg_slot=torch.tensor([2, 0, 3, 1], dtype=torch.int32, device=DEVICE), num_segments=4, max_q_len=max(step))
        out = k.matrix_memory(rows[:, :qk], rows[:, qk:2 * qk], rows[:, 2 * qk:2 * qk + inner], rows[:, at:at + heads],
                              rows[:, at + heads:at + 2 * heads], i_bias.to(DEVICE), f_bias.to(DEVICE), cap, 1e-6,
                              rows[:, 2 * qk + inner:at], weight.to(DEVICE), 1e-5, state, maximum, ctx, heads, dim, vdim, dtype)
        for i in range(4):
            got[i].append(out[first[i]:first[i] + step[i]].float().cpu())
            done[i] += step[i]
    for i in range(4):
        u = sequences[i].double()
        q, kk = u[:, :qk].view(-1, heads, dim) * dim ** -0.5, u[:, qk:2 * qk].view(-1, heads, dim)
        v = u[:, 2 * qk:2 * qk + inner].view(-1, heads, vdim)
        log_in = cap * torch.tanh((u[:, at:at + heads] + i_bias.double()) / cap)
        log_forget = torch.nn.functional.logsigmoid(cap * torch.tanh((u[:, at + heads:at + 2 * heads] + f_bias.double()) / cap))
        want = torch.zeros(total[i], heads, vdim, dtype=F64)
        for h in range(heads):
            want[:, h] = plain.matrix_memory(q[:, h], kk[:, h], v[:, h], log_in[:, h], log_forget[:, h])
        want = plain.rms(want, 1e-5).reshape(total[i], inner) * weight.double() * torch.sigmoid(u[:, 2 * qk + inner:at])
        error = float((torch.cat(got[i]).double() - want).abs().max()) / float(want.abs().max())
        # a head whose numerator nearly cancels is blown up by its norm, rounding and all
        assert error < (1e-4 if dtype == F32 else 1e-2), f"request {i}: off by {error:.2e}"


# ---------------------------------------------------------------- the engine
@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("name", ["MIXED", "ODD", "PLAIN"])
def test_prefill_against_token_by_token(name, dtype):
    config = getattr(zs, name)
    engine = zs.ZuEngine(config, dtype, DEVICE, seed=1)
    tokens = zs.tokens_for(config["vocab"], 75, 8)
    want = engine.plain(tokens)
    for what, cuts in (("whole", []), ("token by token", range(1, 75)), ("prompt then decode", [40] + list(range(41, 75)))):
        zs.assert_logits_close(engine.run_cuts(what, tokens, cuts), want, dtype, what)


@pytest.mark.parametrize("cuts", [[2, 4, 6, 8], [3, 19, 20, 52], [16, 32, 48, 64], [1, 2, 35, 37, 90], [21, 42, 50, 63]])
def test_portions_of_several_sizes(cuts):
    engine = zs.ZuEngine(zs.MIXED, F32, DEVICE, seed=1)
    tokens = zs.tokens_for(131, 100, 9)
    zs.assert_logits_close(engine.run_cuts("a", tokens, cuts), engine.plain(tokens), F32)


def test_float32_logits_do_not_depend_on_the_cut():
    engine = zs.ZuEngine(zs.MIXED, F32, DEVICE, seed=1)
    tokens = zs.tokens_for(131, 90, 10)
    whole = engine.run_cuts("a", tokens, [])
    pieces = engine.run_cuts("b", tokens, [2, 5, 30, 31, 64])
    assert float((whole - pieces).abs().max()) <= 2e-5 * float(whole.abs().max())


def test_the_first_tokens_of_a_sequence():
    engine = zs.ZuEngine(zs.MIXED, F32, DEVICE, seed=14)
    for length in (1, 2, 3, 13):
        tokens = zs.tokens_for(131, length, length)
        want = engine.plain(tokens)
        zs.assert_logits_close(engine.run_cuts("p", tokens, []), want, F32, f"prompt of {length}")
        zs.assert_logits_close(engine.run_cuts("d", tokens, range(1, length)), want, F32, f"decoded from the first token, {length}")


@pytest.mark.parametrize("dtype", DTYPES)
def test_batches_of_unequal_requests(dtype):
    engine = zs.ZuEngine(zs.MIXED, dtype, DEVICE, seed=7, num_pages=40)
    prompts = {"a": zs.tokens_for(131, 70, 1), "b": zs.tokens_for(131, 41, 2), "c": zs.tokens_for(131, 9, 3),
               "d": zs.tokens_for(131, 100, 4)}
    plan = [{"a": 30, "b": 1, "d": 2}, {"a": 1, "b": 16, "c": 9, "d": 50}, {"a": 1, "b": 1, "d": 1},
            {"a": 38, "b": 23, "d": 47}]
    got = engine.run_plan(prompts, plan)
    for name, tokens in prompts.items():
        zs.assert_logits_close(got[name], engine.plain(tokens), dtype, name)


def test_pages_and_slots_are_used_again():
    """Two slots and few pages serve six requests in turn: a slot's memory and maximum start at zero again, pages the
    window has passed are taken by others, and pages written by one request are read by the next."""
    config = zs.config([zs.latent(2, 8, 4, 6, 12), zs.mlstm(2, 8, 12, 8.0, zs.dense(24, 1.0)),
                        zs.attention(4, 2, 6, 10, 11, zs.rotation(100.0, 4)), zs.latent(3, 6, 4, 8, 12, kv_from=0)], width=40, vocab=70)
    slow = {"l1.mix.f.b": lambda t: torch.full_like(t, 7.0), "l1.mix.i.b": lambda t: torch.full_like(t, 5.0)}
    engine = zs.ZuEngine(config, F32, DEVICE, seed=16, page_size=8, num_pages=[14, 8], max_requests=2, max_tokens=64,
                         max_step_tokens=16, overrides=slow)
    for number in range(3):
        prompts = {f"a{number}": zs.tokens_for(70, 33 + 7 * number, 20 + number), f"b{number}": zs.tokens_for(70, 25, 30 + number)}
        plan = []
        for start in range(0, 60, 6):
            step = {name: min(6, len(tokens) - start) for name, tokens in prompts.items() if start < len(tokens)}
            if step:
                plan.append(step)
        got = engine.run_plan(prompts, plan)
        for name, tokens in prompts.items():
            zs.assert_logits_close(got[name], engine.plain(tokens), F32, name)
        engine.cache.check_consistency()
    assert engine.cache.stats().free_pages == (14, 8)


HOWS = {"prompt": lambda query, length: [], "decoded": lambda query, length: [3] + list(range(4, length)),
        "portions": lambda query, length: [2, max(3, query - 1), query, min(query + 2, length)]}


@pytest.mark.parametrize("dtype,dim,kv_heads", [(F32, 48, 1), (BF16, 64, 2)])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portions"])
@pytest.mark.parametrize("query,key,window", [
    (290, 2, 1000),      # a key far back among hundreds
    (271, 15, 300),      # far back, at the last place of a page
    (64, 63, 300),       # the neighbour, across a page's and a tile's border
    (48, 32, 300),       # a page's first place
    (5, 0, 300),         # the very first token
    (299, 150, 150),     # the window's last key
    (299, 149, 150),     # one too far
    (255, 192, 64),      # just inside, windows that end with tiles
    (256, 192, 64),      # just outside
    (131, 125, 7),       # windows shorter than a page
    (131, 124, 7),
    (131, 130, 1),       # it sees itself only
])
def test_far_keys_page_borders_and_window_edges_with_a_dominant_key(query, key, window, how, dtype, dim, kv_heads):
    length = 300
    config, overrides = zs.dominant_key_case(length, query, key, window, seed=query + key, dim=dim, kv_heads=kv_heads)
    engine = zs.ZuEngine(config, dtype, DEVICE, seed=5, overrides=overrides, num_pages=24, max_tokens=320)
    tokens = list(range(length))
    want = engine.plain(tokens)
    got = engine.run_cuts("a", tokens, HOWS[how](query, length))
    zs.assert_logits_close(got[query:query + 1], want[query:query + 1], dtype, f"query {query}")
    zs.assert_logits_close(got, want, dtype)
    # the case tells: with another token at the key's place, the answer at the query differs exactly if it is seen
    hidden = list(tokens)
    hidden[key] = (key + 101) % length
    change = float((engine.plain(hidden)[query] - want[query]).abs().max()) / float(want[query].abs().max())
    if query - key < window:
        assert change > 0.1
    else:
        assert change < 1e-12
        wider = json.loads(json.dumps(config))
        wider["layers"][0]["mixer"]["mask"]["size"] = query - key + 1
        seen = engine.plain(tokens, config_dict=wider)
        assert float((seen[query] - want[query]).abs().max()) > 0.1 * float(want[query].abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
@pytest.mark.parametrize("shared", [False, True])
@pytest.mark.parametrize("how", ["prompt", "decoded", "portions"])
@pytest.mark.parametrize("query,key", [(290, 2), (271, 15), (64, 63), (48, 32), (5, 0), (33, 31), (299, 0)])
def test_far_keys_and_page_borders_through_latents(query, key, how, shared, dtype):
    length = 300
    config, overrides = zs.dominant_latent_case(length, query, key, seed=query + key, shared=shared)
    engine = zs.ZuEngine(config, dtype, DEVICE, seed=5, overrides=overrides, num_pages=24, max_tokens=320)
    tokens = list(range(length))
    want = engine.plain(tokens)
    got = engine.run_cuts("a", tokens, HOWS[how](query, length))
    zs.assert_logits_close(got[query:query + 1], want[query:query + 1], dtype, f"query {query}")
    zs.assert_logits_close(got, want, dtype)
    hidden = list(tokens)
    hidden[key] = (key + 101) % length
    assert float((engine.plain(hidden)[query] - want[query]).abs().max()) > 0.1 * float(want[query].abs().max())


@pytest.mark.parametrize("dtype", DTYPES)
def test_the_sink_shows_where_scores_are_low(dtype):
    """With tiny scores a window of few keys gives the sink a visible share; with large ones next to none."""
    for scale in (1e-3, 3.0):
        config = zs.config([zs.attention(2, 1, 16, 16, 3, zs.rotation(100.0, 8), scale=scale)], width=40, vocab=50)
        engine = zs.ZuEngine(config, dtype, DEVICE, seed=3)
        tokens = zs.tokens_for(50, 40, 2)
        want = engine.plain(tokens)
        zs.assert_logits_close(engine.run_cuts("a", tokens, [20] + list(range(21, 40))), want, dtype)
    q = torch.zeros(4, 2, dtype=F64)
    assert torch.allclose(plain.window_weights(q, q, 1.0, 3).sum(1), torch.tensor([1 / 2, 2 / 3, 3 / 4, 3 / 4], dtype=F64))


@pytest.mark.parametrize("dtype", DTYPES)
def test_long_decoding_through_captured_steps(dtype):
    engine = zs.ZuEngine(zs.MIXED, dtype, DEVICE, seed=14, num_pages=64)
    tokens = zs.tokens_for(131, 260, 13)
    want = engine.plain(tokens)
    got = engine.run_cuts("a", tokens, [30] + list(range(31, 260)))
    assert engine.runner.graph_replays > 100
    zs.assert_logits_close(got, want, dtype)
    other = zs.tokens_for(131, 60, 14)
    engine.cache.create_request("x")
    engine.cache.create_request("y")
    first = engine.step([("x", tokens[:20], range(20)), ("y", other[:10], range(10))])
    rows = {"x": [first[:20]], "y": [first[20:]]}
    for i in range(40):
        logits = engine.step([("x", tokens[20 + i:21 + i], [0]), ("y", other[10 + i:11 + i], [0])])
        rows["x"].append(logits[:1])
        rows["y"].append(logits[1:])
    zs.assert_logits_close(torch.cat(rows["x"]), want[:60], dtype, "x")
    zs.assert_logits_close(torch.cat(rows["y"]), engine.plain(other[:50]), dtype, "y")


@pytest.mark.parametrize("dtype", DTYPES)
def test_sizes_the_tensor_core_kernels_take(dtype):
    engine = zs.ZuEngine(zs.WIDE, dtype, DEVICE, seed=14, num_pages=80, max_tokens=1024)
    tokens = zs.tokens_for(520, 420, 22)
    want = engine.plain(tokens)
    zs.assert_logits_close(engine.run_cuts("a", tokens, [300, 301, 302, 350]), want, dtype)
    prompts = {"p": tokens[:200], "q": zs.tokens_for(520, 150, 24)}
    got = engine.run_plan(prompts, [{"p": 130, "q": 1}, {"p": 1, "q": 140}, {"p": 69, "q": 9}])
    zs.assert_logits_close(got["p"], want[:200], dtype, "p")
    zs.assert_logits_close(got["q"], engine.plain(prompts["q"]), dtype, "q")


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_at_random(seed):
    config = zs.random_config(seed + 100)
    for dtype in DTYPES:
        engine = zs.ZuEngine(config, dtype, DEVICE, seed=seed, num_pages=40)
        prompts = {"a": zs.tokens_for(config["vocab"], 45, seed), "b": zs.tokens_for(config["vocab"], 21, seed + 50)}
        got = engine.run_plan(prompts, [{"a": 17, "b": 1}, {"a": 1, "b": 2}, {"a": 2, "b": 18}, {"a": 25}])
        for name, tokens in prompts.items():
            zs.assert_logits_close(got[name], engine.plain(tokens), dtype, f"seed {seed} {name}", spread=8e-2)


def test_greedy_generation_through_the_scheduler():
    parts = zs.ZuEngine(zs.MIXED, F32, DEVICE, seed=31)
    engine = ContinuousBatchEngine.from_model(parts.model, block_size=8, total_blocks=96, max_running_requests=3,
                                              max_batch_tokens=24, max_model_len=160)
    prompts = [zs.tokens_for(131, length, 40 + i) for i, length in enumerate([5, 37, 18, 50, 2])]
    generated = engine.generate(prompts, max_new_tokens=12)
    for prompt, got in zip(prompts, generated):
        sequence = list(prompt)
        for _ in range(12):
            sequence.append(int(torch.argmax(parts.plain(sequence)[-1])))
        assert got == sequence[len(prompt):]


def test_command_line_and_replay_program_with_a_model_folder(tmp_path):
    """``make-random`` writes a Zugarax folder from a config.json, ``generate`` reproduces the plain
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

    (tmp_path / "config.json").write_text(json.dumps(zs.MIXED))
    folder = tmp_path / "model"
    cli("-m", "mini_llm_runtime_b200", "make-random", "--config", str(tmp_path / "config.json"), "--seed", "4",
        "--out", str(folder))
    tensors = read_checkpoint(folder)
    prompt = zs.tokens_for(131, 11, 6)
    sequence = list(prompt)
    for _ in range(5):
        sequence.append(int(torch.argmax(plain.forward(zs.MIXED, tensors, sequence)[0][-1])))
    record = json.loads(cli("-m", "mini_llm_runtime_b200", "generate", "--model", str(folder), "--dtype", "float32",
                            "--max-model-len", "64", "--prompt-ids", ",".join(map(str, prompt)), "--max-new-tokens", "5"
                            ).splitlines()[-1])
    assert record["generated_ids"] == sequence[len(prompt):]

    other = zs.tokens_for(131, 30, 7)
    steps = [{"step": 0, "entries": [{"id": "p", "tokens": prompt[:4], "want": [0, 3]}], "end": []},
             {"step": 1, "entries": [{"id": "p", "tokens": prompt[4:], "want": [6]},
                                     {"id": "o", "tokens": other, "want": [29]}], "end": ["p"]},
             {"step": 2, "entries": [], "end": ["o"]}]
    out = cli(os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out",
              str(tmp_path / "logits"), "--max-tokens", "64", stdin="\n".join(json.dumps(s) for s in steps) + "\n")
    assert [line for line in out.splitlines() if line.startswith("done")] == ["done 0", "done 1", "done 2"]
    first = torch.from_numpy(np.fromfile(tmp_path / "logits" / "0.f32", dtype="<f4").reshape(2, 131))
    second = torch.from_numpy(np.fromfile(tmp_path / "logits" / "1.f32", dtype="<f4").reshape(2, 131))
    want = plain.forward(zs.MIXED, tensors, prompt)[0]
    zs.assert_logits_close(torch.cat([first, second[:1]]), want[[0, 3, 10]], F32)
    zs.assert_logits_close(second[1:], plain.forward(zs.MIXED, tensors, other)[0][29:], F32)
