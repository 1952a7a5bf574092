"""``bench.py --arch vetevik``: the Vetevik architecture at layer sizes that resemble real models, beside
Ratilorn (the engine's closest model: a recurrence behind a short convolution, an attention of its own kind,
a 32-bit stream, routed experts) at equal width, depth, heads, state sizes and experts.

Per size: a 2,048-token prefill and decode steps at batch 8 around a context of 2,048 tokens, both models with
random weights in bfloat16, timed on the device (CUDA events, median of the regions; weights and caches
together exceed the L2).  Then each kernel that Vetevik adds or extends, alone, with the bytes or flops it must
move and the fraction of the measured roofline that makes, next to the like kernel of an existing model.  One
JSON line.
"""

from __future__ import annotations

import json
import sys

import bench_bopilorn
import bench_ratilorn
import bench_zazasun as common
from bench_zazasun import PREFILL, Bench, _segments, _time, model_points

SIZES = {
    # groups of (delta, delta, attention) layers; the recurrence as wide as the model
    "896": dict(width=896, groups=4, vocab=32000, heads=14, kv_heads=2, dim=64, chunk=4096,
                delta=dict(heads=14, kv_heads=7, dim=64, vdim=64), experts=16, top=2, ff=2432),
    "2048": dict(width=2048, groups=4, vocab=32000, heads=16, kv_heads=4, dim=128, chunk=4096,
                 delta=dict(heads=32, kv_heads=16, dim=128, vdim=64), experts=64, top=6, ff=1408),
}
TAPS, NORM_GROUPS, SOFTCAP = 4, 4, 50.0


def vetevik_config(size):
    from mini_llm_runtime_b200.config import config_from_dict

    s = SIZES[size]
    mlp = {"kind": "moe", "expert": {"ff": s["ff"]}, "router": {"experts": s["experts"], "top": s["top"]}}
    attention = {"heads": s["heads"], "kv_heads": s["kv_heads"], "dim": s["dim"], "vdim": s["dim"], "scale": s["dim"] ** -0.5,
                 "softcap": SOFTCAP, "mask": {"size": s["chunk"]}}
    delta = {"type": "delta", "mixer": {**s["delta"], "conv": TAPS}, "mlp": mlp}
    group = [delta, delta, {"type": "attention", "mixer": attention, "mlp": mlp}]
    return config_from_dict({"architecture": "Vetevik", "vocab": s["vocab"], "width": s["width"],
                             "norm": {"eps": 1e-6, "groups": NORM_GROUPS}, "residual_mult": 0.5,
                             "max_positions": common.MAX_POSITIONS, "layers": group * s["groups"]})


def _pieces(size):
    s = SIZES[size]
    width, d = s["width"], s["delta"]
    attention = (2 * s["heads"] + s["kv_heads"]) * s["dim"] * width + width * s["heads"] * s["dim"]
    inner = d["heads"] * d["vdim"]
    delta = (2 * d["kv_heads"] * d["dim"] + 2 * inner + 2 * d["heads"]) * width + width * inner
    return s, width, attention, delta, 3 * width * s["ff"], s["experts"] * width


def vetevik_numbers(size, batch=8):
    """Bytes a decode step of `batch` rows must read and flops of a prefill, from the sizes."""
    s, width, attention, delta, expert, router = _pieces(size)
    layers, attention_layers, delta_layers = 3 * s["groups"], s["groups"], 2 * s["groups"]
    touched = bench_bopilorn.experts_touched(s["experts"], s["top"], batch)
    mixers = attention_layers * attention + delta_layers * delta
    head = s["vocab"] * width
    d = s["delta"]
    state = d["heads"] * d["vdim"] * d["dim"]

    def sequence_flops(rows, before=0):
        pairs = rows * before + rows * (rows + 1) // 2      # the chunk is longer than the prompt
        return attention_layers * pairs * s["heads"] * 4 * s["dim"] + delta_layers * rows * state * 7

    return {"weight_bytes": int(2 * (mixers + layers * (2 * router + touched * expert) + head)),
            "kv_bytes_per_token": attention_layers * s["kv_heads"] * s["dim"] * 2,
            "cache_bytes_per_request": delta_layers * 2 * 4 * state,
            "linear_flops_per_token": 2 * (mixers + layers * (router + s["top"] * expert)), "head_flops_per_row": 2 * head,
            "attention_flops": sequence_flops}


def prefill_weight_bytes(size):
    s, width, attention, delta, expert, router = _pieces(size)
    return int(2 * (s["groups"] * attention + 2 * s["groups"] * delta
                    + 3 * s["groups"] * (2 * router + s["experts"] * expert) + s["vocab"] * width))


def _ratilorn_size(size):
    """Ratilorn at the same sizes under a name of its own: no shared expert, no groups of experts to choose among."""
    s = SIZES[size]
    name = size + "v"
    bench_ratilorn.SIZES[name] = dict(
        width=s["width"], groups=s["groups"], vocab=s["vocab"], heads=s["heads"], kv_heads=s["kv_heads"], dim=s["dim"],
        ssm=dict(heads=s["delta"]["heads"], vdim=s["delta"]["vdim"], state=s["delta"]["dim"]), experts=s["experts"],
        top=s["top"], ff=s["ff"], router_groups=(1, 1), shared=0)
    return name


def kernel_points(size, peak):
    """Each new or extended kernel alone: 2,048 rows of one request (prefill) and 8 requests of one row (decode)."""
    import torch

    from mini_llm_runtime_b200 import ops
    from mini_llm_runtime_b200.ops.cuda_ops import AttentionBatch, plan_attention

    k = ops.current()
    s = SIZES[size]
    width, heads, kv_heads, dim = s["width"], s["heads"], s["kv_heads"], s["dim"]
    d = s["delta"]
    qk, inner = d["kv_heads"] * d["dim"], d["heads"] * d["vdim"]
    channels, state_size = 2 * qk + inner, d["heads"] * d["vdim"] * d["dim"]
    flush = torch.zeros(96 << 20, dtype=torch.float32, device="cuda")      # 384 MB, three times the L2
    bf16, f32 = torch.bfloat16, torch.float32
    hbm = peak["hbm_gbs"] * 1e9
    out = {}

    def record(name, micros, nbytes=None, flops=None):
        entry = {"us": round(micros, 2)}
        if nbytes is not None:
            entry["bytes"] = int(nbytes)
            entry["hbm_frac"] = round(nbytes / (micros * 1e-6) / hbm, 4) if micros > 0 else None
        if flops is not None:
            entry["tflops"] = round(flops / (micros * 1e-6) / 1e12, 3) if micros > 0 else None
            entry["bf16_peak_frac"] = round(flops / (micros * 1e-6) / (peak["bf16_tflops"] * 1e12), 5) if micros > 0 else None
        out[name] = entry

    vector = lambda n: torch.randn(n, device="cuda")      # noqa: E731
    cases = {"prefill": _segments([PREFILL], [0]), "decode": _segments([1] * 8, [2047] * 8)}
    for label, ctx in cases.items():
        rows = int(ctx.lengths.sum())
        page, context = 16, int(ctx.positions.max() + ctx.lengths.max())
        pages_per_request = -(-context // page)
        table = torch.arange(ctx.num_segments * pages_per_request, dtype=torch.int32, device="cuda").view(ctx.num_segments, -1)
        k_pool = torch.randn(ctx.num_segments * pages_per_request, kv_heads, page, dim, device="cuda").to(bf16)
        v_pool = torch.randn_like(k_pool)
        slots = torch.cat([torch.arange(int(p), int(p) + int(c), dtype=torch.int64) + i * pages_per_request * page
                           for i, (p, c) in enumerate(zip(ctx.positions, ctx.lengths))]).cuda()
        arrays, counts = plan_attention(ctx.lengths, ctx.positions)
        arrays = {name: torch.from_numpy(value).cuda() for name, value in arrays.items()}
        batch = AttentionBatch(ctx.seg_q_start, ctx.seg_q_len, ctx.seg_pos0, ctx.seg_slot, table, ctx.num_segments,
                               ctx.max_q_len, context, arrays, counts)
        projected = (torch.randn(rows, (2 * heads + kv_heads) * dim, device="cuda") * 0.2).to(bf16)
        q, key, gate = (projected[:, :heads * dim], projected[:, heads * dim:(heads + kv_heads) * dim],
                        projected[:, (heads + kv_heads) * dim:])
        pairs = sum(int(p) + i + 1 for p, c in zip(ctx.positions, ctx.lengths) for i in range(int(c)))
        key_bytes = context * ctx.num_segments * kv_heads * dim * 2
        row_bytes = rows * heads * dim * 2
        slopes, sink = torch.rand(heads, device="cuda") * 0.01, vector(heads)
        record(f"shaped_attention.{label}",
               _time(lambda: k.shaped_attention(q, key, None, slots, k_pool, None, batch, heads, kv_heads, dim, dim, dim ** -0.5,
                                                softcap=SOFTCAP, slopes=slopes, chunk=s["chunk"], sink=sink, gate=gate), flush),
               key_bytes + 3 * row_bytes, pairs * heads * 4 * dim)
        q_plain = q.contiguous()
        r1, r2, pb = torch.rand(heads, device="cuda"), torch.rand(heads, device="cuda"), vector(heads)
        talk = torch.eye(heads, device="cuda") + 0.1 * torch.randn(heads, heads, device="cuda")
        record(f"ratilorn.sigmoid_attention.{label}",
               _time(lambda: k.sigmoid_attention(q_plain, k_pool, v_pool, batch, heads, kv_heads, dim, dim, dim ** -0.5,
                                                 distance=(r1, r2), score_bias=pb, head_mix=talk), flush),
               2 * key_bytes + 2 * row_bytes, pairs * heads * 4 * dim)
        record(f"ratilorn.softmax_attention.{label}",
               _time(lambda: k.paged_attention(q_plain, k_pool, v_pool, batch, heads, kv_heads, dim, dim ** -0.5, None), flush),
               2 * key_bytes + 2 * row_bytes, pairs * heads * 4 * dim)
        # the delta rule: convolution, recurrence, gated head norm; beside the state-space recurrence of equal sizes
        wide = channels + inner + 2 * d["heads"]
        wide += -wide % 8
        rows32 = torch.randn(rows, wide, device="cuda") * 0.5
        conv = torch.randn(channels, TAPS, device="cuda") * 0.3
        conv_state = torch.zeros(8, TAPS - 1, channels, device="cuda")
        record(f"causal_conv.{label}", _time(lambda: k.causal_conv(rows32[:, :channels], conv, None, conv_state, ctx), flush),
               rows * channels * 8 + (2 * ctx.num_segments * (TAPS - 1) * channels * 4 if label == "decode" else 0))
        mixed = k.causal_conv(rows32[:, :channels], conv, None, conv_state, ctx)
        dt_bias, a_log = vector(d["heads"]) * 0.1, -torch.rand(d["heads"], device="cuda")
        state = torch.zeros(8, d["heads"], d["vdim"], d["dim"], device="cuda")
        at = channels + inner
        state_bytes = 2 * ctx.num_segments * state_size * 4
        record(f"delta_rule_scan.{label}",
               _time(lambda: k.delta_rule_scan(mixed[:, :qk], mixed[:, qk:2 * qk], mixed[:, 2 * qk:], rows32[:, at:at + d["heads"]],
                                               rows32[:, at + d["heads"]:at + 2 * d["heads"]], dt_bias, a_log, state, ctx,
                                               d["heads"], d["kv_heads"], d["dim"], d["vdim"], 1e-6), flush),
               rows * (2 * qk + 2 * inner + 2 * d["heads"]) * 4 + state_bytes, rows * state_size * 7)
        n = d["dim"]
        skip = vector(d["heads"])
        B, C, x = (torch.randn(rows, m, device="cuda") * 0.5 for m in (n, n, inner))
        dt_raw = torch.randn(rows, d["heads"], device="cuda")
        record(f"ratilorn.state_space_scan.{label}",
               _time(lambda: k.state_space_scan(x, B, C, dt_raw, dt_bias, a_log, skip, state, ctx, d["heads"], d["vdim"], n, 1), flush),
               rows * (inner * 8 + 2 * n * 4 + d["heads"] * 4) + state_bytes, rows * state_size * 4)
        y, head_weight = torch.randn(rows, inner, device="cuda"), torch.ones(d["vdim"], device="cuda")
        record(f"gated_head_norm.{label}",
               _time(lambda: k.gated_head_norm(y, rows32[:, channels:at], head_weight, 1e-6, d["heads"], bf16), flush), rows * inner * 10)
        norm_weight = torch.ones(inner, device="cuda")
        record(f"ratilorn.gated_group_norm.{label}",
               _time(lambda: k.gated_group_norm(y, rows32[:, channels:at], norm_weight, 1e-6, 1, bf16), flush), rows * inner * 10)
        # the stream: x += norm(delta) and the next norm of x, in parts of the row
        stream, delta_rows = torch.randn(rows, width, device="cuda"), torch.randn(rows, width, device="cuda")
        w1, w2 = torch.ones(width, device="cuda"), torch.ones(width, device="cuda")
        for name, groups in (("rms_norm_step", NORM_GROUPS), ("ratilorn.rms_norm_step", 1)):
            record(f"{name}.{label}",
                   _time(lambda: k.rms_norm_step(stream, 1e-6, delta=delta_rows, delta_weight=w1, norm_weight=w2, out_dtype=bf16,
                                                 groups=groups), flush), rows * width * 14)
        # the experts, weighed at their inputs and at their outputs
        experts, top, ff = s["experts"], s["top"], s["ff"]
        h = torch.randn(rows, width, device="cuda").to(bf16)
        gate_up = (torch.randn(experts, 2 * ff, width, device="cuda") * 0.02).to(bf16)
        down = (torch.randn(experts, width, ff, device="cuda") * 0.02).to(bf16)
        chosen = torch.rand(rows, experts, device="cuda").topk(top, dim=1).indices.to(torch.int32)
        weights = torch.rand(rows, top, device="cuda")
        touched = experts if label == "prefill" else bench_bopilorn.experts_touched(experts, top, rows)
        expert_bytes = touched * 3 * width * ff * 2 + rows * width * 6
        for name, at_input in (("experts_weighed_at_input", True), ("ratilorn.experts", False)):
            record(f"{name}.{label}",
                   _time(lambda: k.routed_experts(h, chosen, weights, gate_up, down, 64, "silu", weigh_input=at_input), flush),
                   expert_bytes, rows * top * 6 * width * ff)
        del k_pool, v_pool, gate_up, down
        torch.cuda.empty_cache()
    k.raise_if_device_error()
    return out


def run(args, host):
    import torch

    if not torch.cuda.is_available():
        print(json.dumps({"error": "no CUDA device"}))
        return 1
    peak = host.peaks()
    record = {"metric": "Vetevik beside Ratilorn at equal sizes: prefill of 2,048 tokens and decode at batch 8",
              "dtype": "bf16", "data": "synthetic (seeded random weights and token ids)", "n_gpus": 1,
              "context": 2048, "peaks": peak, "sizes": {}, "kernels": {}}
    with host.ClockSampler() as clocks:
        for size in SIZES:
            entry = {}
            other = _ratilorn_size(size)
            for name, config, numbers, weights in (
                    ("vetevik", vetevik_config(size), vetevik_numbers(size), prefill_weight_bytes(size)),
                    ("ratilorn", bench_ratilorn.ratilorn_config(other), bench_ratilorn.ratilorn_numbers(other),
                     bench_ratilorn.prefill_weight_bytes(other))):
                bench = Bench(f"{name} {size}", config, numbers, host)
                entry[name] = model_points(bench, host, args, peak)
                entry[name]["layers"] = len(bench.model.blocks)
                flops = entry[name]["prefill_frac_of_bf16_peak"] * peak["bf16_tflops"] * 1e12 * entry[name]["prefill_2048_ms"] / 1e3
                bound_ms = max(flops / (peak["bf16_tflops"] * 1e12), weights / (peak["hbm_gbs"] * 1e9)) * 1e3
                entry[name]["prefill_roofline_ms"] = round(bound_ms, 3)
                entry[name]["prefill_frac_of_roofline"] = round(bound_ms / entry[name]["prefill_2048_ms"], 4)
                bench.close()
            record["sizes"][size] = entry
            record["kernels"][size] = kernel_points(size, peak)
            print(f"[bench] {size}: {json.dumps(entry)}", file=sys.stderr)
            print(f"[bench] {size} kernels: {json.dumps(record['kernels'][size])}", file=sys.stderr)
    record["clocks"] = clocks.summary()
    print(json.dumps(record))
    return 0
