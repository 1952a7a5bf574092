"""``bench.py --arch zugarax``: the Zugarax architecture at layer sizes that resemble real models, beside Rozesun
(the engine's closest model: attention over latents, a clamped gated feed-forward, a 32-bit stream) at equal width,
depth, feed-forward and latent sizes.

Per size: a 2,048-token prefill and decode steps at batch 8 around a context of 2,048 tokens, both models with
random weights in bfloat16, timed on the device (CUDA events, median of the regions; weights and caches
together exceed the L2).  Then each kernel that Zugarax adds or extends, alone, with the bytes or flops it must
move and the fraction of the measured roofline that makes, next to the like kernel of an existing model: the
windowed attention beside Vetevik's (keys that are values) and the plain softmax attention, the matrix memory beside
Vetevik's delta rule with equal states, the latent attention beside Rozesun's (the same kernel; a latent read by a second
layer costs no kernel), the prepare kernel beside Bopilorn's.  One JSON line.
"""

from __future__ import annotations

import json
import math
import sys

import bench_rozesun
import bench_zazasun as common
from bench_zazasun import PREFILL, Bench, _segments, _time, model_points

SIZES = {
    # groups of (latent, windowed attention, matrix memory) layers; every second latent layer reads the one before it
    "896": dict(attention=dict(heads=14, kv_heads=2, dim=64, vdim=64), mlstm=dict(heads=7, dim=128, vdim=128)),
    "2048": dict(attention=dict(heads=16, kv_heads=4, dim=128, vdim=128), mlstm=dict(heads=16, dim=128, vdim=128)),
}
WINDOW, LIMIT, CAP = 1024, 7.0, 15.0
RAMP = {"factor": 4.0, "original": 4096, "fast": 32.0, "slow": 1.0}
BANDS = {"factor": 8.0, "original": 8192, "low": 1.0, "high": 4.0}


def _sizes(size):
    s = bench_rozesun.SIZES[size]
    return {**SIZES[size], "width": s["width"], "ff": s["ff"], "groups": s["groups"], "vocab": s["vocab"],
            "latent": {name: s["mixer"][name] for name in ("heads", "dim", "rot_dim", "vdim", "kv_rank")}}


def zugarax_config(size):
    from mini_llm_runtime_b200.config import config_from_dict

    s = _sizes(size)
    mlp = {"kind": "dense", "ff": s["ff"], "limit": LIMIT}
    lat, att = s["latent"], s["attention"]
    latent = dict(lat, rot={"base": 10000.0, "dims": lat["rot_dim"], "scaling": RAMP}, scale=1.0 / math.sqrt(lat["dim"] + lat["rot_dim"]))
    attention = dict(att, mask={"size": WINDOW}, scale=att["dim"] ** -0.5, rot={"base": 5e5, "dims": att["dim"] // 2, "scaling": BANDS})
    layers = []
    for group in range(s["groups"]):
        shared = {"kv_from": 3 * (group - 1)} if group % 2 else {}
        layers += [{"type": "latent_attention", "mixer": {**latent, **shared}, "mlp": mlp},
                   {"type": "attention", "mixer": attention, "mlp": mlp},
                   {"type": "mlstm", "mixer": dict(s["mlstm"], gate_cap=CAP), "mlp": mlp}]
    return config_from_dict({"architecture": "Zugarax", "vocab": s["vocab"], "width": s["width"],
                             "max_positions": common.MAX_POSITIONS, "norm": {"eps": 1e-6}, "embedding": {"scale": 1.0},
                             "logit_softcap": 30.0, "layers": layers})


def zugarax_numbers(config, context):
    """Bytes a decode step must read (and write: the memory's state) and flops of a prefill, from the configuration."""
    width = config.width
    matrices = cache_bytes = 0
    terms = []
    for layer in config.layers:
        a = layer.mixer_args
        if layer.type == "latent_attention":
            own = 0 if "kv_from" in a else a["kv_rank"] + a["rot_dim"]
            matrices += (a["heads"] * (a["dim"] + a["rot_dim"]) + own + a["heads"] * a["vdim"]) * width
            matrices += a["heads"] * (a["dim"] + a["vdim"]) * a["kv_rank"]
            cache_bytes += context * (a["kv_rank"] + a["rot_dim"]) * 2
        elif layer.type == "attention":
            matrices += (a["heads"] * (a["dim"] + 2 * a["vdim"]) + a["kv_heads"] * (a["dim"] + a["vdim"])) * width
            cache_bytes += min(context, a["window"]) * a["kv_heads"] * (a["dim"] + a["vdim"]) * 2
        else:
            matrices += (2 * a["heads"] * a["dim"] + 3 * a["heads"] * a["vdim"] + 2 * a["heads"]) * width
            cache_bytes += 2 * 4 * a["heads"] * (a["vdim"] + 1) * a["dim"]
        matrices += 3 * width * layer.mlp_args["ff"]
        terms.append((layer.type, a))

    def sequence_flops(rows):
        total = 0
        for kind, a in terms:
            if kind == "latent_attention":
                total += rows * (rows + 1) // 2 * a["heads"] * 2 * (2 * a["kv_rank"] + a["rot_dim"])
            elif kind == "attention":
                total += sum(min(p + 1, a["window"]) for p in range(rows)) * a["heads"] * 2 * (a["dim"] + a["vdim"])
            else:
                total += rows * a["heads"] * (a["vdim"] + 1) * a["dim"] * 5
        return total

    head = config.vocab * width
    return {"weight_bytes": 2 * (matrices + head), "kv_bytes_per_token": 0, "cache_bytes_per_request": cache_bytes,
            "linear_flops_per_token": 2 * matrices, "head_flops_per_row": 2 * head,
            "attention_flops": lambda rows, before=0: sequence_flops(rows)}


def kernel_points(size, peak):
    """Each new or extended kernel alone: 2,048 rows of one request (prefill) and 8 requests of one row (decode)."""
    import torch

    from mini_llm_runtime_b200 import ops
    from mini_llm_runtime_b200.ops.cuda_ops import AttentionBatch, plan_attention

    k = ops.current()
    s = _sizes(size)
    width, att, mem, lat = s["width"], s["attention"], s["mlstm"], s["latent"]
    heads, kv_heads, dim, vdim = att["heads"], att["kv_heads"], att["dim"], att["vdim"]
    flush = torch.zeros(96 << 20, dtype=torch.float32, device="cuda")      # 384 MB, three times the L2
    bf16 = torch.bfloat16
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

    cases = {"prefill": _segments([PREFILL], [0]), "decode": _segments([1] * 8, [2047] * 8)}
    for label, ctx in cases.items():
        rows = int(ctx.lengths.sum())
        page, context = 16, int(ctx.positions.max() + ctx.lengths.max())
        pages_per_request = -(-context // page)
        table = torch.arange(ctx.num_segments * pages_per_request, dtype=torch.int32, device="cuda").view(ctx.num_segments, -1)
        pool_pages = ctx.num_segments * pages_per_request
        k_pool = torch.randn(pool_pages, kv_heads, page, dim, device="cuda").to(bf16)
        v_pool = torch.randn(pool_pages, kv_heads, page, vdim, device="cuda").to(bf16)
        positions = torch.cat([torch.arange(int(p), int(p) + int(n), dtype=torch.int32)
                               for p, n in zip(ctx.positions, ctx.lengths)]).cuda()
        slots = torch.cat([torch.arange(int(p), int(p) + int(c), dtype=torch.int64) + i * pages_per_request * page
                           for i, (p, c) in enumerate(zip(ctx.positions, ctx.lengths))]).cuda()
        arrays, counts = plan_attention(ctx.lengths, ctx.positions)
        arrays = {name: torch.from_numpy(value).cuda() for name, value in arrays.items()}
        batch = AttentionBatch(ctx.seg_q_start, ctx.seg_q_len, ctx.seg_pos0, ctx.seg_slot, table, ctx.num_segments,
                               ctx.max_q_len, context, arrays, counts)
        # the windowed attention, with and without its window, beside Vetevik's and the plain softmax attention
        sizes = (heads * dim, kv_heads * dim, kv_heads * vdim, heads * vdim)
        projected = (torch.randn(rows, sum(sizes), device="cuda") * 0.2).to(bf16)
        q, key, value, gate = projected.split(sizes, dim=1)
        q_plain = q.contiguous()
        sink = torch.zeros(heads, device="cuda")
        row_bytes = rows * heads * (dim + 2 * vdim) * 2

        def visible(window):
            pairs = sum(min(int(p) + i + 1, window) for p, c in zip(ctx.positions, ctx.lengths) for i in range(int(c)))
            keys = sum(min(int(p) + int(c), window + int(c) - 1) for p, c in zip(ctx.positions, ctx.lengths))
            return pairs, keys

        for name, window in (("windowed_attention", WINDOW), ("windowed_attention.all_keys", 1 << 30)):
            pairs, keys = visible(window)
            record(f"{name}.{label}",
                   _time(lambda: k.shaped_attention(q_plain, None, None, slots, k_pool, v_pool, batch, heads, kv_heads, dim, vdim,
                                                    dim ** -0.5, window=0 if window > context else window, sink=sink, gate=gate,
                                                    write_kv=False), flush),
                   keys * kv_heads * (dim + vdim) * 2 + row_bytes, pairs * heads * 2 * (dim + vdim))
            record(f"vetevik.shaped_attention{name[18:]}.{label}",
                   _time(lambda: k.shaped_attention(q_plain, None, None, slots, k_pool, None, batch, heads, kv_heads, dim, vdim,
                                                    dim ** -0.5, window=0 if window > context else window, softcap=50.0, sink=sink,
                                                    gate=gate, write_kv=False), flush),
                   keys * kv_heads * dim * 2 + row_bytes, pairs * heads * 2 * (dim + vdim))
            record(f"qwen.attention{name[18:]}.{label}",
                   _time(lambda: k.paged_attention(q_plain, k_pool, v_pool, batch, heads, kv_heads, dim, dim ** -0.5,
                                                   None if window > context else window), flush),
                   keys * kv_heads * (dim + vdim) * 2 + rows * heads * (dim + vdim) * 2, pairs * heads * 2 * (dim + vdim))
        # norm, rotation and cache write, beside Bopilorn's (32-bit projections, norms over whole projections)
        weight, freq = torch.ones(dim, device="cuda"), torch.rand(dim // 4, device="cuda")
        record(f"head_prepare.{label}",
               _time(lambda: k.head_prepare(q, key, value, positions, weight, weight, 1e-6, freq, 1.0, False, slots, k_pool, v_pool,
                                            heads, kv_heads, dim, vdim), flush), rows * sum(sizes[:3]) * 4)
        wide = torch.randn(rows, sum(sizes[:3]), device="cuda")
        wq, wk = torch.ones(heads * dim, device="cuda"), torch.ones(kv_heads * dim, device="cuda")
        record(f"bopilorn.rotated_prepare.{label}",
               _time(lambda: k.rotated_prepare(wide, positions, wq, wk, 1e-6, freq, 1.0, None, False, False, slots, k_pool, v_pool,
                                               heads, kv_heads, dim, vdim), flush), rows * sum(sizes[:3]) * 6)
        # latent attention and what stands around it
        rank, rot, lheads = lat["kv_rank"], lat["rot_dim"], lat["heads"]
        pool = torch.randn(pool_pages, 1, page, rank + rot, device="cuda").to(bf16)
        q_width = lheads * (lat["dim"] + rot)
        down = torch.randn(rows, q_width + rank + rot, device="cuda")
        wc, lfreq = torch.ones(rank, device="cuda"), torch.rand(rot // 2, device="cuda")
        record(f"latent_prepare.{label}",
               _time(lambda: k.latent_prepare(down, 0, 0, q_width, rank, rot, None, wc, 1e-6, positions, lfreq, True, slots, pool,
                                              magnitude=1.2), flush), rows * (rank + rot) * 6)
        w_uk = (torch.randn(lheads * lat["dim"], rank, device="cuda") * 0.05).to(bf16)
        record(f"absorb_queries.{label}",
               _time(lambda: k.absorb_queries(down[:, :q_width], w_uk, lheads, lat["dim"], rot, rank, positions, lfreq, True, 1.2), flush),
               rows * lheads * ((lat["dim"] + rot) * 4 + (rank + rot) * 2) + w_uk.numel() * 2, 2 * rows * lheads * lat["dim"] * rank)
        qa = (torch.randn(rows, lheads * (rank + rot), device="cuda") * 0.2).to(bf16)
        pairs, keys = visible(1 << 30)
        record(f"latent_attention.{label}",
               _time(lambda: k.latent_attention(qa, pool, batch, lheads, rank, rot, 0.08, 0, None), flush),
               keys * (rank + rot) * 2 + rows * lheads * ((rank + rot) * 2 + rank * 4), pairs * lheads * 2 * (2 * rank + rot))
        mixed = torch.randn(rows, lheads * rank, device="cuda")
        w_uv = (torch.randn(lheads * lat["vdim"], rank, device="cuda") * 0.05).to(bf16)
        record(f"latent_values.{label}",
               _time(lambda: k.latent_values(mixed, w_uv, lheads, lat["vdim"], rank, None, False), flush),
               rows * lheads * (rank * 4 + lat["vdim"] * 2) + w_uv.numel() * 2, 2 * rows * lheads * lat["vdim"] * rank)
        # the matrix memory (all of its kernels) beside the delta rule of equal states (with its head norm)
        mh, md, mv = mem["heads"], mem["dim"], mem["vdim"]
        qk, inner = mh * md, mh * mv
        total = 2 * qk + 2 * inner + 2 * mh
        rows32 = torch.randn(rows, total + -total % 8, device="cuda") * 0.5
        bias, memory_weight = torch.zeros(mh, device="cuda"), torch.ones(inner, device="cuda")
        state, maximum = torch.zeros(8, mh, mv + 1, md, device="cuda"), torch.zeros(8, mh, device="cuda")
        at = 2 * qk + 2 * inner
        state_bytes = 2 * ctx.num_segments * mh * mv * md * 4
        memory = lambda: k.matrix_memory(rows32[:, :qk], rows32[:, qk:2 * qk], rows32[:, 2 * qk:2 * qk + inner],      # noqa: E731
                                         rows32[:, at:at + mh], rows32[:, at + mh:at + 2 * mh], bias, bias + 3, CAP, 1e-6,
                                         rows32[:, 2 * qk + inner:at], memory_weight, 1e-6, state, maximum, ctx, mh, md, mv, bf16)
        record(f"matrix_memory.{label}", _time(memory, flush), rows * (2 * qk + 2 * inner + 2 * mh) * 4 + rows * inner * 2 + state_bytes,
               rows * mh * mv * md * 5)
        delta_state, head_weight = torch.zeros(8, mh, mv, md, device="cuda"), torch.ones(mv, device="cuda")

        def delta():
            y = k.delta_rule_scan(rows32[:, :qk], rows32[:, qk:2 * qk], rows32[:, 2 * qk:2 * qk + inner], rows32[:, at:at + mh],
                                  rows32[:, at + mh:at + 2 * mh], bias, bias, delta_state, ctx, mh, mh, md, mv, 1e-6)
            return k.gated_head_norm(y, rows32[:, 2 * qk + inner:at], head_weight, 1e-6, mh, bf16)

        record(f"vetevik.delta_rule_and_norm.{label}", _time(delta, flush),
               rows * (2 * qk + 2 * inner + 2 * mh) * 4 + rows * inner * 2 + state_bytes, rows * mh * mv * md * 7)
        # the stream's step, the gate with and without biases, the logits' cap
        stream, rows_in, w = torch.randn(rows, width, device="cuda"), torch.randn(rows, width, device="cuda"), torch.ones(width, device="cuda")
        record(f"add_and_rms_norm.{label}",
               _time(lambda: k.rms_norm_step(stream, 1e-6, norm_weight=w, out_dtype=bf16, offset=rows_in), flush), rows * width * 14)
        lnw = (w, torch.zeros_like(w))
        record(f"rozesun.add_layer_norm_layer_norm.{label}",
               _time(lambda: k.layer_norm_step(stream, 1e-6, delta=rows_in, delta_norm=lnw, norm=lnw, out_dtype=bf16), flush),
               rows * width * 14)
        h = torch.randn(rows, width, device="cuda").to(bf16)
        gate_up = (torch.randn(2 * s["ff"], width, device="cuda") * 0.02).to(bf16)
        gate_bias = torch.randn(2 * s["ff"], device="cuda").to(bf16)
        for name, b in (("gate_up_with_biases", gate_bias), ("rozesun.gate_up", None)):
            record(f"{name}.{label}", _time(lambda: k.linear_clamped_gate(h, gate_up, 64, LIMIT, 1.702, bias=b), flush),
                   gate_up.numel() * 2 + rows * (width + s["ff"]) * 2, 2 * rows * gate_up.numel())
        logits = torch.randn(min(rows, 8), s["vocab"], device="cuda")
        record(f"softcap.{label}", _time(lambda: k.softcap_(logits, 30.0), flush), logits.numel() * 8)
        record(f"rozesun.scale.{label}", _time(lambda: k.scale_(logits, 1.001), flush), logits.numel() * 8)
        del k_pool, v_pool, pool, gate_up
        torch.cuda.empty_cache()
    k.raise_if_device_error()
    return out


def run(args, host):
    import torch

    if not torch.cuda.is_available():
        print(json.dumps({"error": "no CUDA device"}))
        return 1
    peak = host.peaks()
    record = {"metric": "Zugarax beside Rozesun at equal sizes: prefill of 2,048 tokens and decode at batch 8",
              "dtype": "bf16", "data": "synthetic (seeded random weights and token ids)", "n_gpus": 1,
              "window": WINDOW, "context": 2048, "peaks": peak, "sizes": {}, "kernels": {}}
    with host.ClockSampler() as clocks:
        for size in SIZES:
            entry = {}
            for name, config, numbers in (
                    ("zugarax", zugarax_config(size), zugarax_numbers), ("rozesun", bench_rozesun.rozesun_config(size), bench_rozesun.rozesun_numbers)):
                bench = Bench(f"{name} {size}", config, numbers(config, 2048), host)
                entry[name] = model_points(bench, host, args, peak)
                entry[name]["layers"] = len(bench.model.blocks)
                bench.close()
            record["sizes"][size] = entry
            record["kernels"][size] = kernel_points(size, peak)
            print(f"[bench] {size}: {json.dumps(entry)}", file=sys.stderr)
            print(f"[bench] {size} kernels: {json.dumps(record['kernels'][size])}", file=sys.stderr)
    record["clocks"] = clocks.summary()
    print(json.dumps(record))
    return 0
